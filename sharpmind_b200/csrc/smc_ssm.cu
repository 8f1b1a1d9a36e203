// State-space (Mamba-2) sequence mixing between its two projections:
//   x | B | C pass a causal convolution per channel and SiLU;  dt = softplus(dt_raw + bias)
//   S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t        per head, S [state, vdim]
//   o = RMSNorm in parts(y * SiLU(z)) * w
// Two forms of the recurrence: token after token (ssm_scan_kernel: decoding, short portions, fp32, odd sizes), and chunks of
// 64 tokens whose inner sums are matrix products on the tensor cores (ssm_chunk_kernel).
// dt, decays, S and y are fp32.  A sequence's state is S and the inputs of the convolution's last taps (position p in row
// p % taps of its ring).
#include <cuda_bf16.h>

#include <type_traits>

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

// ------------------------------------------------------------------------------ recurrence in chunks (bfloat16 inputs)
// With c_t the running sum of log decays inside a chunk and S the state before it,
//   y_t = sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s  +  exp(c_t) S^T C_t  +  D x_t
//   S'  = exp(c_end) S + sum_s exp(c_end - c_s) dt_s B_s x_s^T
// x, B and C are bfloat16 already; every fp32 factor (weights of the first sum, the state, the scaled x) enters its product
// as a pair hi + lo of bfloat16, i.e. with 16 bits, and all sums are fp32.  The log decays are summed in double.  One CTA
// carries 32 value columns of one head through the whole portion, the state in accumulator registers.
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void *src, bool in)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
// {a, b} as bfloat16 pairs: hi, and lo = what hi leaves
__device__ __forceinline__ void split2(float a, float b, uint32_t &hi, uint32_t &lo)
{
    const bf16 ah = __float2bfloat16_rn(a), bh = __float2bfloat16_rn(b);
    const __nv_bfloat162 h = __halves2bfloat162(ah, bh), l = __floats2bfloat162_rn(a - __bfloat162float(ah), b - __bfloat162float(bh));
    hi = *reinterpret_cast<const uint32_t *>(&h), lo = *reinterpret_cast<const uint32_t *>(&l);
}

constexpr int CQ = 64, CP = 32;
struct ChunkSmem {  // byte offsets; rows are padded to an odd number of 16-byte units
    int ldn, cb, x, m, xw, st, f, total;
};
__host__ __device__ inline ChunkSmem chunk_smem(int N)
{
    ChunkSmem o;
    const int n16 = (N + 15) & ~15;
    o.ldn = (n16 + 8) * 2;
    o.cb = 0;                                   // two buffers of C [64][N] then B [64][N]
    o.x = o.cb + 4 * CQ * o.ldn;                // two buffers of x [64][32]
    o.m = o.x + 2 * CQ * 80;                    // weights hi, lo [64][64]
    o.xw = o.m + 2 * CQ * 144;                  // scaled x hi, lo [64][32]
    o.st = o.xw + 2 * CQ * 80;                  // state hi, lo [32][N]
    o.f = o.st + 2 * CP * o.ldn;                // dt, c, exp(c) [64] fp32 each, then exp(c_end)
    o.total = o.f + 3 * CQ * 4 + 16;
    return o;
}

template <int NTW>  // state tiles of 8 columns per warp (four warps across N)
__global__ void __launch_bounds__(256) ssm_chunk_kernel(const bf16 *__restrict__ xbc, const float *__restrict__ dt_raw, float *__restrict__ y,
                                                        float *__restrict__ state, smc_rows rw, const float *__restrict__ dt_bias,
                                                        const float *__restrict__ a_log, const float *__restrict__ d_skip, int heads, int P, int N,
                                                        int groups)
{
    extern __shared__ __align__(16) uint8_t csm[];
    const ChunkSmem L = chunk_smem(N);
    const uint32_t sb = (uint32_t)__cvta_generic_to_shared(csm);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int h = blockIdx.x, p0 = blockIdx.y * CP, grp = h / (heads / groups), T = rw.n;
    const int inner = heads * P, ch = inner + 2 * groups * N, n16 = (N + 15) & ~15;
    float *s_dt = reinterpret_cast<float *>(csm + L.f), *s_c = s_dt + CQ, *s_ec = s_c + CQ, *s_end = s_ec + CQ;
    for (int e = threadIdx.x; e < L.total / 16; e += 256) reinterpret_cast<uint4 *>(csm)[e] = make_uint4(0u, 0u, 0u, 0u);
    smc_grid_dep_sync();
    __syncthreads();
    const bool fresh = rw.pos[rw.seq0] == 0;
    float *st = state + ((size_t)rw.seq0 * heads + h) * P * N;
    const float A = -expf(a_log[h]), D = d_skip[h], bias = dt_bias[h];
    const int cn = N / 8, cx = min(CP, P - p0) / 8, per = 2 * cn + cx;
    auto fetch = [&](int t0, int buf) {
        for (int e = threadIdx.x; e < CQ * per; e += 256) {
            const int t = e / per, c = e % per;
            const bool in = t0 + t < T;
            const bf16 *src = xbc + (size_t)(in ? t0 + t : T - 1) * ch;
            if (c < cn) cp16(sb + L.cb + (uint32_t)((2 * buf * CQ + t) * L.ldn + 16 * c), src + inner + (groups + grp) * N + 8 * c, in);
            else if (c < 2 * cn) cp16(sb + L.cb + (uint32_t)(((2 * buf + 1) * CQ + t) * L.ldn + 16 * (c - cn)), src + inner + grp * N + 8 * (c - cn), in);
            else cp16(sb + L.x + (uint32_t)((buf * CQ + t) * 80 + 16 * (c - 2 * cn)), src + h * P + p0 + 8 * (c - 2 * cn), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    // state accumulators: rows p (16 per warp pair member), columns n
    const int sm_m = warp & 1, sm_n = warp >> 1;  // 16-row tile of the 32 columns of x, quarter of N
    float S[NTW][4];
    const int nt_per = (n16 / 8 + 3) / 4;
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
        S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
        const int n = (sm_n * nt_per + i) * 8 + 2 * tg, pa = p0 + sm_m * 16 + g;
        if (fresh || i >= nt_per || n >= N) continue;
        if (pa < P) S[i][0] = st[(size_t)pa * N + n], S[i][1] = st[(size_t)pa * N + n + 1];
        if (pa + 8 < P) S[i][2] = st[(size_t)(pa + 8) * N + n], S[i][3] = st[(size_t)(pa + 8) * N + n + 1];
    }
    auto put_state = [&]() {
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n = (sm_n * nt_per + i) * 8 + 2 * tg;
            if (i >= nt_per || n >= n16) continue;
            uint32_t hi, lo;
            uint8_t *d = csm + L.st + (sm_m * 16 + g) * L.ldn + 2 * n;
            split2(S[i][0], S[i][1], hi, lo);
            *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CP * L.ldn) = lo;
            split2(S[i][2], S[i][3], hi, lo);
            d += 8 * L.ldn;
            *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CP * L.ldn) = lo;
        }
    };
    put_state();
    // ldmatrix lane offsets: A operand rows / B operand [n][k] rows, two tiles / transposed [k][n]
    const int la = (lane & 7) + 8 * ((lane >> 3) & 1), lah = 16 * (lane >> 4);
    const int lb = (lane & 7) + 8 * (lane >> 4), lbh = 16 * ((lane >> 3) & 1);
    const int mt = warp & 3, nh = warp >> 2;      // 16-token tile, half of the other side
    int buf = 0;
    for (int t0 = 0; t0 < T; t0 += CQ, buf ^= 1) {
        if (t0 + CQ < T) {
            fetch(t0 + CQ, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        if (warp == 0) {  // step sizes and running log decays of the chunk: two tokens per lane
            float dt[2];
            double a[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int t = t0 + 2 * lane + i;
                dt[i] = t < T ? softplus(dt_raw[(size_t)t * heads + h] + bias) : 0.f;  // past the end: no input, no decay
                a[i] = (double)(A * dt[i]);
            }
            double sum = a[0] + a[1];
            for (int d = 1; d < 32; d <<= 1) {
                const double v = __shfl_up_sync(0xffffffffu, sum, d);
                if (lane >= d) sum += v;
            }
            const float c0 = (float)(sum - a[1]), c1 = (float)sum;
            s_dt[2 * lane] = dt[0], s_dt[2 * lane + 1] = dt[1];
            s_c[2 * lane] = c0, s_c[2 * lane + 1] = c1;
            s_ec[2 * lane] = expf(c0), s_ec[2 * lane + 1] = expf(c1);
            if (lane == 31) *s_end = c1;
        }
        __syncthreads();
        const uint32_t cC = sb + L.cb + (uint32_t)(2 * buf * CQ * L.ldn), cB = cC + (uint32_t)(CQ * L.ldn), cX = sb + L.x + (uint32_t)(buf * CQ * 80);
        // ---- weights of the first sum: C_t . B_s for 16 tokens x 32 sources per warp
        float G[4][4], Y[2][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i) Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
        const bool any = 32 * nh <= 16 * mt + 15;  // else every source lies after every token
        for (int k = 0; k < n16 / 16; ++k) {
            uint32_t a[4], b[4], sh[4], sl[4];
            ldsm4(cC + (uint32_t)((16 * mt + la) * L.ldn + 32 * k + lah), a);
            if (any) {
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    ldsm4(cB + (uint32_t)((32 * nh + 16 * j + lb) * L.ldn + 32 * k + lbh), b);
                    mma_bf16(G[2 * j], a, b[0], b[1]);
                    mma_bf16(G[2 * j + 1], a, b[2], b[3]);
                }
            }
            // ---- S^T C: 16 tokens x 16 value columns per warp
            ldsm4(sb + L.st + (uint32_t)((16 * nh + lb) * L.ldn + 32 * k + lbh), sh);
            ldsm4(sb + L.st + (uint32_t)((CP + 16 * nh + lb) * L.ldn + 32 * k + lbh), sl);
            mma_bf16(Y[0], a, sl[0], sl[1]), mma_bf16(Y[1], a, sl[2], sl[3]);
            mma_bf16(Y[0], a, sh[0], sh[1]), mma_bf16(Y[1], a, sh[2], sh[3]);
        }
        {
            const int ta = 16 * mt + g, tb = ta + 8;
            const float ca = s_c[ta], cb = s_c[tb];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int s = 32 * nh + 8 * i + 2 * tg;
                float w[4];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    w[j] = s + j <= ta ? G[i][j] * (expf(ca - s_c[s + j]) * s_dt[s + j]) : 0.f;
                    w[2 + j] = s + j <= tb ? G[i][2 + j] * (expf(cb - s_c[s + j]) * s_dt[s + j]) : 0.f;
                }
                uint32_t hi, lo;
                uint8_t *d = csm + L.m + ta * 144 + 2 * s;
                split2(w[0], w[1], hi, lo);
                *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CQ * 144) = lo;
                split2(w[2], w[3], hi, lo);
                d += 8 * 144;
                *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CQ * 144) = lo;
            }
            const float ea = s_ec[ta], eb = s_ec[tb];
#pragma unroll
            for (int i = 0; i < 2; ++i) Y[i][0] *= ea, Y[i][1] *= ea, Y[i][2] *= eb, Y[i][3] *= eb;
        }
        // ---- x scaled for the state update
        const float end = *s_end;
        for (int e = threadIdx.x; e < CQ * CP / 2; e += 256) {
            const int t = e >> 4, c = (e & 15) * 2;
            const float f = expf(end - s_c[t]) * s_dt[t];
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162 *>(csm + L.x + (buf * CQ + t) * 80 + 2 * c);
            uint32_t hi, lo;
            split2(__bfloat162float(v.x) * f, __bfloat162float(v.y) * f, hi, lo);
            *reinterpret_cast<uint32_t *>(csm + L.xw + t * 80 + 2 * c) = hi, *reinterpret_cast<uint32_t *>(csm + L.xw + (CQ + t) * 80 + 2 * c) = lo;
        }
        __syncthreads();
        // ---- y: weights x x, sources up to the tile's last token
        for (int k = 0; k <= mt; ++k) {
            uint32_t ah[4], al[4], b[4];
            ldsm4(sb + L.m + (uint32_t)((16 * mt + la) * 144 + 32 * k + lah), ah);
            ldsm4(sb + L.m + (uint32_t)((CQ + 16 * mt + la) * 144 + 32 * k + lah), al);
            ldsm4t(cX + (uint32_t)((16 * k + la) * 80 + 32 * nh + lah), b);
            mma_bf16(Y[0], al, b[0], b[1]), mma_bf16(Y[1], al, b[2], b[3]);
            mma_bf16(Y[0], ah, b[0], b[1]), mma_bf16(Y[1], ah, b[2], b[3]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int c = 16 * nh + 8 * i + 2 * tg;
            if (p0 + c >= P) continue;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int t = 16 * mt + g + 8 * j;
                if (t0 + t >= T) continue;
                const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162 *>(csm + L.x + (buf * CQ + t) * 80 + 2 * c);
                *reinterpret_cast<float2 *>(y + (size_t)(t0 + t) * inner + h * P + p0 + c) =
                    make_float2(fmaf(D, __bfloat162float(v.x), Y[i][2 * j]), fmaf(D, __bfloat162float(v.y), Y[i][2 * j + 1]));
            }
        }
        // ---- state
        const float dec = expf(end);
#pragma unroll
        for (int i = 0; i < NTW; ++i) S[i][0] *= dec, S[i][1] *= dec, S[i][2] *= dec, S[i][3] *= dec;
#pragma unroll
        for (int k = 0; k < CQ / 16; ++k) {
            // A operand stored [token][column]: transposed load, matrices in the order (k, m): (0,0) (0,8) (8,0) (8,8)
            uint32_t ah[4], al[4];
            const uint32_t off = (uint32_t)((16 * k + (lane & 7) + 8 * (lane >> 4)) * 80 + 32 * sm_m + 16 * ((lane >> 3) & 1));
            ldsm4t(sb + L.xw + off, ah);
            ldsm4t(sb + L.xw + (uint32_t)(CQ * 80) + off, al);
#pragma unroll
            for (int i = 0; i < NTW; i += 2) {
                const int nt = sm_n * nt_per + i;
                if (i >= nt_per || nt * 8 >= n16) continue;
                uint32_t b[4];
                // two tiles; the second may lie past this warp's share: its product is then not used
                ldsm4t(cB + (uint32_t)((16 * k + la) * L.ldn + 16 * nt + (nt * 8 + 8 < n16 ? lah : 0)), b);
                mma_bf16(S[i], al, b[0], b[1]), mma_bf16(S[i], ah, b[0], b[1]);
                if (i + 1 < nt_per) mma_bf16(S[i + 1], al, b[2], b[3]), mma_bf16(S[i + 1], ah, b[2], b[3]);
            }
        }
        __syncthreads();  // everybody has read the state planes, the weights and this chunk's buffers
        put_state();
    }
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
        const int n = (sm_n * nt_per + i) * 8 + 2 * tg, pa = p0 + sm_m * 16 + g;
        if (i >= nt_per || n >= N) continue;
        if (pa < P) *reinterpret_cast<float2 *>(st + (size_t)pa * N + n) = make_float2(S[i][0], S[i][1]);
        if (pa + 8 < P) *reinterpret_cast<float2 *>(st + (size_t)(pa + 8) * N + n) = make_float2(S[i][2], S[i][3]);
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

// portions from this many rows on are taken in chunks
constexpr int CHUNK_ROWS = 32;

template <typename T>
int recur_chunks(smc_ctx *ctx, const smc_ssm_dims &d, const smc_ssm_bufs &b, const smc_rows &rw, const float *dt_bias, const float *a_log,
                 const float *d_skip, cudaStream_t s)
{
    if constexpr (!std::is_same<T, bf16>::value) return SMC_E_UNSUPPORTED;
    const ChunkSmem L = chunk_smem(d.state);
    if (d.vdim % 8 || d.state % 8 || d.state > 256 || L.total > 220 * 1024) return SMC_E_UNSUPPORTED;
    auto go = [&](auto kernel) {
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(d.heads, (d.vdim + CP - 1) / CP), dim3(256), (size_t)L.total, s, (const bf16 *)b.xbc, b.dt_raw, b.y,
                       b.state, rw, dt_bias, a_log, d_skip, d.heads, d.vdim, d.state, d.groups);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    if (d.state <= 64) return go(ssm_chunk_kernel<2>);
    if (d.state <= 128) return go(ssm_chunk_kernel<4>);
    return go(ssm_chunk_kernel<8>);
}

template <typename T>
int recur_steps(smc_ctx *ctx, const smc_ssm_dims &d, const smc_ssm_bufs &b, const smc_rows &rw, const float *dt_bias, const float *a_log,
                const float *d_skip, cudaStream_t s)
{
    const bool seq = rw.seq0 >= 0;
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
    return SMC_OK;
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
    int rc = seq && rw.n >= CHUNK_ROWS ? recur_chunks<T>(ctx, d, b, rw, dt_bias, a_log, d_skip, s) : SMC_E_UNSUPPORTED;
    if (rc == SMC_E_UNSUPPORTED) rc = recur_steps<T>(ctx, d, b, rw, dt_bias, a_log, d_skip, s);
    if (rc) return rc;
    const size_t nsm = (size_t)(inner / d.norm_groups) * sizeof(float);
    if (nsm > 40 * 1024) SMC_CUDA(ctx, cudaFuncSetAttribute(ssm_gate_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)nsm));
    smc_launch_dep(ctx->use_pdl, ssm_gate_norm_kernel<T>, dim3(rw.n, d.norm_groups), dim3(128), nsm, s, (const float *)b.y, static_cast<const T *>(b.zx),
                   b.ld, norm, static_cast<T *>(b.o), inner, d.norm_groups, d.eps);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

}  // namespace

int smc_ssm_mix(smc_ctx *ctx, const smc_ssm_dims &d, const smc_ssm_bufs &b, const smc_rows &rw, int is_bf16, const float *conv_w, const float *conv_b,
                const float *dt_bias, const float *a_log, const float *d_skip, const float *norm, cudaStream_t s)
{
    if (is_bf16) return mix<bf16>(ctx, d, b, rw, conv_w, conv_b, dt_bias, a_log, d_skip, norm, s);
    return mix<float>(ctx, d, b, rw, conv_w, conv_b, dt_bias, a_log, d_skip, norm, s);
}
