// Matmuls over dense bfloat16 weights:  out[m, n] = sum_k x[m, k] * w[n, k],  w [N, K] row-major.
//
//   dense_skinny_kernel   bfloat16 rows, up to 32 of them per pass: weights stream from global memory straight into
//                         mma.sync fragments (16 weight rows per CTA, K split over its warps), bound by HBM
//   dense_tc_kernel       bfloat16 rows at prompt sizes: tiled TMA -> swizzled shared memory -> tcgen05.mma -> TMEM,
//                         persistent, 128 tokens x 128 or 256 weight rows per tile
//   dense_rows_kernel     fp32 (or odd-shaped bfloat16) rows, up to eight: a warp per weight row, fp32 FMAs
//   dense_tile_kernel     fp32 (or odd-shaped bfloat16) rows, more: 64 x 64 tiles, fp32 FMAs
//
// fp32 rows are multiplied in true fp32 (a bfloat16 weight widens exactly).  Every kernel shares one epilogue: plain
// fp32 or bfloat16 columns, a second fp32 destination for the trailing columns, or act(gate) * up of woven row pairs; before
// that a bias, SiLU over a range of columns or a soft cap, and a sum into what the destination holds.
#include <type_traits>

#include "smc_mma.cuh"
#include "smc_tc.cuh"

namespace {

// gelu_tanh(z) = z / (1 + e^(-2u)), u = sqrt(2/pi) (z + 0.044715 z^3): 1 + tanh u is 2 / (1 + e^(-2u))
__device__ __forceinline__ float gelu_arg(float z) { return -1.5957691216057308f * z * fmaf(0.044715f * z, z, 1.0f); }
__device__ __forceinline__ float act_pair(int woven, float gate, float up)
{
    return (woven == 2 ? __fdiv_rn(gate, 1.0f + expf(gelu_arg(gate))) : silu(gate)) * up;
}
// in front of a bfloat16 rounding
template <bool GELU>
__device__ __forceinline__ float act_pair_fast(float gate, float up)
{
    return __fdividef(gate, 1.0f + __expf(GELU ? gelu_arg(gate) : -gate)) * up;
}
// what happens to a sum before it is stored
__device__ __forceinline__ float finish(const smc_dense_out &o, int n, float v)
{
    if (o.bias) v += o.bias[n];
    if (n >= o.silu_from && n < o.silu_to) v = o.y_bf16 ? silu_for<bf16>(v) : silu(v);
    if (o.softcap > 0.f) v = o.softcap * tanhf(__fdiv_rn(v, o.softcap));
    return v;
}
__device__ __forceinline__ void put(const smc_dense_out &o, int m, int n, float v)
{
    v = finish(o, n, v);
    if (o.split > 0 && n >= o.split) o.y32[(size_t)m * o.ld32 + (n - o.split)] = v;
    else if (o.y_bf16) static_cast<bf16 *>(o.y)[(size_t)m * o.ldy + n] = __float2bfloat16_rn(v);
    else {
        float *y = static_cast<float *>(o.y) + (size_t)m * o.ldy + n;
        *y = o.accumulate ? *y + v : v;
    }
}
__device__ __forceinline__ void put_pair(const smc_dense_out &o, int m, int i, float gate, float up)
{
    const float v = act_pair(o.woven, gate, up);
    if (o.y_bf16) static_cast<bf16 *>(o.y)[(size_t)m * o.ldy + i] = __float2bfloat16_rn(v);
    else static_cast<float *>(o.y)[(size_t)m * o.ldy + i] = v;
}

// ------------------------------------------------------------------------------ few rows, bfloat16
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1)
{
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// One CTA: 16 weight rows, NT * 8 activation rows, eight warps that take every eighth 32-element chunk of K.  The
// contraction does not care which k a fragment register holds as long as both operands agree, so lane (g, q) takes the
// 16 contiguous bytes k = 32 c + 8 q .. + 7 of weight rows g and g + 8 and of activation row g: every load is 16 bytes
// wide and a row's four lanes read 64 contiguous bytes.  The first weight chunks are requested before the kernel waits
// for its predecessor.  Grouped form (blockIdx.z = group): N rows per group, each group with its own columns of x.
// HALF: eight weight rows per CTA (the upper half of each fragment is zero), for matrices with too few rows to fill the SMs.
// KV > 0: one fp32 row of up to 1024 KV elements instead of x, layer-normed by every CTA while its first weights arrive.
struct NormedRow {
    const float *x, *w;
    float eps;
};
template <int KV>
__device__ __forceinline__ void stage_normed(const NormedRow &r, int K, bf16 *xs)
{
    __shared__ float red[2][8];
    float4 v[KV], g[KV];
    float sum = 0.f, ss = 0.f;
#pragma unroll
    for (int j = 0; j < KV; ++j) {
        const int i = threadIdx.x + 256 * j;
        v[j] = 4 * i < K ? reinterpret_cast<const float4 *>(r.x)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        g[j] = 4 * i < K ? __ldg(reinterpret_cast<const float4 *>(r.w) + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    auto block = [&](float t, float *s) {
        t = smc_group_sum<32>(t);
        if ((threadIdx.x & 31) == 0) s[threadIdx.x >> 5] = t;
        __syncthreads();
        return ((s[0] + s[1]) + (s[2] + s[3])) + ((s[4] + s[5]) + (s[6] + s[7]));
    };
#pragma unroll
    for (int j = 0; j < KV; ++j) sum += (v[j].x + v[j].y) + (v[j].z + v[j].w);
    const float mean = __fdiv_rn(block(sum, red[0]), (float)K);
#pragma unroll
    for (int j = 0; j < KV; ++j) {
        if (4 * (threadIdx.x + 256 * j) >= K) continue;
        v[j].x -= mean, v[j].y -= mean, v[j].z -= mean, v[j].w -= mean;
        ss = fmaf(v[j].x, v[j].x, ss), ss = fmaf(v[j].y, v[j].y, ss), ss = fmaf(v[j].z, v[j].z, ss), ss = fmaf(v[j].w, v[j].w, ss);
    }
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(block(ss, red[1]), (float)K) + r.eps));
#pragma unroll
    for (int j = 0; j < KV; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (4 * i < K)
            *reinterpret_cast<uint2 *>(xs + 4 * i) = make_uint2(pack2((v[j].x * inv) * g[j].x, (v[j].y * inv) * g[j].y),
                                                                pack2((v[j].z * inv) * g[j].z, (v[j].w * inv) * g[j].w));
    }
    __syncthreads();
}
template <int NT, int U, bool HALF, int KV = 0>
__global__ void __launch_bounds__(256) dense_skinny_kernel(const bf16 *__restrict__ w, const bf16 *__restrict__ x, int ldx, int M, int N, int K,
                                                           smc_dense_out o, int x_group, NormedRow row)
{
    __shared__ __align__(16) bf16 xs[KV ? 1024 * KV : 8];
    constexpr int TOK = NT * 8, ROWS = HALF ? 8 : 16;
    __shared__ float red[8][ROWS][TOK + 1];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, q = lane & 3;
    const int n0 = blockIdx.x * ROWS, m0 = blockIdx.y * TOK, grp0 = blockIdx.z * N;
    const int chunks = (K + 31) >> 5;
    w += (size_t)grp0 * K, x += (size_t)blockIdx.z * x_group;
    const bf16 *w0 = w + (size_t)min(n0 + g, N - 1) * K + 8 * q, *w1 = w + (size_t)min(n0 + g + 8, N - 1) * K + 8 * q;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    uint4 a0[U], a1[U];
    auto fetch = [&](int c0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = c0 + 8 * u;
            const bool in = c < chunks && 32 * c + 8 * q < K;
            a0[u] = in ? smc_ldg_stream16(w0 + 32 * c) : zero;
            a1[u] = in && !HALF ? smc_ldg_stream16(w1 + 32 * c) : zero;
        }
    };
    fetch(warp);
    smc_grid_dep_sync();
    if constexpr (KV > 0) stage_normed<KV>(row, K, xs);
    float acc[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
    for (int c0 = warp; c0 < chunks; c0 += 8 * U) {
        uint4 b0[U], b1[U];
#pragma unroll
        for (int u = 0; u < U; ++u) b0[u] = a0[u], b1[u] = a1[u];
        uint4 xv[U][NT];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int k = 32 * (c0 + 8 * u) + 8 * q;
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                const int m = m0 + 8 * t + g;
                if (KV) xv[u][t] = m == 0 && k < K ? *reinterpret_cast<const uint4 *>(xs + k) : zero;
                else xv[u][t] = m < M && k < K ? *reinterpret_cast<const uint4 *>(x + (size_t)m * ldx + k) : zero;
            }
        }
        fetch(c0 + 8 * U);
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                mma_bf16(acc[t], b0[u].x, b1[u].x, b0[u].y, b1[u].y, xv[u][t].x, xv[u][t].y);
                mma_bf16(acc[t], b0[u].z, b1[u].z, b0[u].w, b1[u].w, xv[u][t].z, xv[u][t].w);
            }
    }
    // accumulator: rows g (0, 1) and g + 8 (2, 3), tokens 2q, 2q + 1
#pragma unroll
    for (int t = 0; t < NT; ++t) {
        red[warp][g][8 * t + 2 * q] = acc[t][0], red[warp][g][8 * t + 2 * q + 1] = acc[t][1];
        if (!HALF) red[warp][g + ROWS - 8][8 * t + 2 * q] = acc[t][2], red[warp][g + ROWS - 8][8 * t + 2 * q + 1] = acc[t][3];
    }
    __syncthreads();
    auto total = [&](int r, int t) {
        float v = red[0][r][t];
#pragma unroll
        for (int i = 1; i < 8; ++i) v += red[i][r][t];
        return v;
    };
    if (o.woven) {
        for (int e = threadIdx.x; e < ROWS / 2 * TOK; e += 256) {
            const int i = e % (ROWS / 2), t = e / (ROWS / 2);
            if (m0 + t < M && n0 + 2 * i + 1 < N) put_pair(o, m0 + t, (n0 >> 1) + i, total(2 * i, t), total(2 * i + 1, t));
        }
    } else {
        for (int e = threadIdx.x; e < ROWS * TOK; e += 256) {
            const int r = e % ROWS, t = e / ROWS;
            if (m0 + t < M && n0 + r < N) put(o, m0 + t, grp0 + n0 + r, total(r, t));
        }
    }
}

// ------------------------------------------------------------------------------ fp32 on the CUDA cores
// A warp per weight row (per row pair when woven), up to eight activation rows.
template <typename TX>
__global__ void __launch_bounds__(256) dense_rows_kernel(const bf16 *__restrict__ w, const TX *__restrict__ x, int ldx, int M, int N, int K,
                                                         smc_dense_out o)
{
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, wid = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int per = o.woven ? 2 : 1;
    if (wid * per >= N) return;
    const int m0 = blockIdx.y * 8, mc = min(8, M - m0);
    float acc[2][8];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int m = 0; m < 8; ++m) acc[j][m] = 0.f;
    for (int k = lane; k < K; k += 32) {
        const float wa = to_f(w[(size_t)wid * per * K + k]);
        const float wb = per == 2 ? to_f(w[((size_t)wid * 2 + 1) * K + k]) : 0.f;
#pragma unroll
        for (int m = 0; m < 8; ++m)
            if (m < mc) {
                const float xv = to_f(x[(size_t)(m0 + m) * ldx + k]);
                acc[0][m] = fmaf(xv, wa, acc[0][m]);
                if (per == 2) acc[1][m] = fmaf(xv, wb, acc[1][m]);
            }
    }
#pragma unroll
    for (int m = 0; m < 8; ++m) {
        const float va = smc_group_sum<32>(acc[0][m]), vb = smc_group_sum<32>(acc[1][m]);
        if (lane == 0 && m < mc) {
            if (per == 2) put_pair(o, m0 + m, wid, va, vb);
            else put(o, m0 + m, wid, va);
        }
    }
}

// 64 x 64 tile, 256 threads with 4 x 4 outputs each (thread column j holds weight rows 4 j .. 4 j + 3: whole pairs).
template <typename TX>
__global__ void __launch_bounds__(256) dense_tile_kernel(const bf16 *__restrict__ w, const TX *__restrict__ x, int ldx, int M, int N, int K,
                                                         smc_dense_out o)
{
    constexpr int KS = 16;
    __shared__ float sx[KS][64 + 4], sw[KS][64 + 4];
    smc_grid_dep_sync();
    const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += KS) {
        for (int e = threadIdx.x; e < 64 * KS; e += 256) {
            const int r = e / KS, c = e % KS;
            sx[c][r] = m0 + r < M && k0 + c < K ? to_f(x[(size_t)(m0 + r) * ldx + k0 + c]) : 0.f;
            sw[c][r] = n0 + r < N && k0 + c < K ? to_f(w[(size_t)(n0 + r) * K + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < KS; ++c) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = sx[c][4 * ty + i], b[i] = sw[c][4 * tx + i];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + 4 * ty + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + 4 * tx + j;
            if (n >= N) continue;
            if (!o.woven) put(o, m, n, acc[i][j]);
            else if (!(j & 1)) put_pair(o, m, n >> 1, acc[i][j], acc[i][j + 1 < 4 ? j + 1 : j]);
        }
    }
}

// ------------------------------------------------------------------------------ prompt sizes: tcgen05
constexpr int TC_M = 128, TC_K = 64;
template <int BN>
struct TcShape {
    static constexpr int STAGES = BN == 256 ? 4 : 5;
    static constexpr uint32_t A_BYTES = TC_M * TC_K * 2, B_BYTES = BN * TC_K * 2, STAGE = A_BYTES + B_BYTES;
    static constexpr uint32_t OFF_BAR = STAGES * STAGE, SMEM = OFF_BAR + 256 + 1024;  // + slack to align the base to 1024
    static constexpr uint32_t COLS = 2 * BN;                                       // two accumulators
};

// What the epilogue does: store (or sum), SiLU or GELU of woven pairs, or everything `finish` knows.
enum { EPI_STORE, EPI_SILU_PAIRS, EPI_GELU_PAIRS, EPI_FINISH };
// y[0..3] += v without waiting for y: every element has one writer per launch, so the result does not depend on an order
__device__ __forceinline__ void add4(float *y, float a, float b, float c, float d)
{
    asm volatile("red.global.add.v4.f32 [%0], {%1, %2, %3, %4};" ::"l"(y), "f"(a), "f"(b), "f"(c), "f"(d) : "memory");
}

// Warp 0: TMA loads; warp 1: MMA issue; warps 2 .. 5: epilogue (one TMEM lane = one token per thread).
template <int BN, int EPI>
__global__ void __launch_bounds__(192, 1) dense_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, int M,
                                                          int N, int K, smc_dense_out o, int *status)
{
    using S = TcShape<BN>;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smc_smem_u32(smem_raw), sbase = (raw + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - raw);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    auto full = [&](int i) { return sbase + S::OFF_BAR + 8u * (uint32_t)i; };
    auto empty = [&](int i) { return sbase + S::OFF_BAR + 8u * (uint32_t)(S::STAGES + i); };
    auto acc_full = [&](int i) { return sbase + S::OFF_BAR + 8u * (uint32_t)(2 * S::STAGES + i); };
    auto acc_empty = [&](int i) { return sbase + S::OFF_BAR + 8u * (uint32_t)(2 * S::STAGES + 2 + i); };
    constexpr uint32_t OFF_PTR = S::OFF_BAR + 8u * (2 * S::STAGES + 4);
    volatile uint32_t *abort_flag = reinterpret_cast<volatile uint32_t *>(smem + OFF_PTR + 4);

    // Tensor memory is taken only after the predecessor has completed, and the successor may start only after it was
    // taken: kernels that overlap on an SM can then never wait for one another's columns.
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (threadIdx.x == 0) {
        for (int i = 0; i < S::STAGES; ++i) smc_mbar_init(full(i), 1), smc_mbar_init(empty(i), 1);
        for (int i = 0; i < 2; ++i) smc_mbar_init(acc_full(i), 1), smc_mbar_init(acc_empty(i), 4);
        *abort_flag = 0;
        smc_fence_barrier_init();
    }
    if (warp == 0) {
        __syncwarp();
        smc_tc_alloc(sbase + OFF_PTR, S::COLS);
    }
    smc_tc_fence_before();
    __syncthreads();
    smc_tc_fence_after();
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(smem + OFF_PTR);

    const int mt = (M + TC_M - 1) / TC_M, nt = (N + BN - 1) / BN, tiles = mt * nt, ksteps = (K + TC_K - 1) / TC_K;
    if (warp == 0) {
        if (lane == 0) {
            int st = 0;
            uint32_t ph = 1;
            for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
                const int m0 = (t % mt) * TC_M, n0 = (t / mt) * BN;
                for (int k = 0; k < ksteps; ++k) {
                    smc_tc_wait(empty(st), ph, abort_flag, status);
                    smc_mbar_expect_tx(full(st), S::STAGE);
                    smc_tma_2d(sbase + (uint32_t)st * S::STAGE, &map_x, k * TC_K, m0, full(st));
                    smc_tma_2d(sbase + (uint32_t)st * S::STAGE + S::A_BYTES, &map_w, k * TC_K, n0, full(st));
                    if (++st == S::STAGES) st = 0, ph ^= 1;
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t IDESC = smc_tc_idesc_bf16(TC_M, BN);
            int st = 0, n = 0;
            uint32_t ph = 0;
            for (int t = blockIdx.x; t < tiles; t += gridDim.x, ++n) {
                const int buf = n & 1;
                smc_tc_wait(acc_empty(buf), (uint32_t)(((n >> 1) & 1) ^ 1), abort_flag, status);
                smc_tc_fence_after();
                const uint32_t d = tmem + (uint32_t)(buf * BN);
                for (int k = 0; k < ksteps; ++k) {
                    smc_tc_wait(full(st), ph, abort_flag, status);
                    smc_tc_fence_after();
                    const uint64_t da = smc_tc_desc_sw128(sbase + (uint32_t)st * S::STAGE), db = smc_tc_desc_sw128(sbase + (uint32_t)st * S::STAGE + S::A_BYTES);
#pragma unroll
                    for (int kk = 0; kk < TC_K / 16; ++kk) smc_tc_mma(d, da + 2 * kk, db + 2 * kk, IDESC, (k | kk) != 0 ? 1u : 0u);
                    smc_tc_commit(empty(st));
                    if (++st == S::STAGES) st = 0, ph ^= 1;
                }
                smc_tc_commit(acc_full(buf));
            }
        }
    } else {
        const int quarter = warp & 3;
        int n = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x, ++n) {
            const int buf = n & 1, m = (t % mt) * TC_M + quarter * 32 + lane, n0 = (t / mt) * BN;
            if (lane == 0) smc_tc_wait(acc_full(buf), (uint32_t)((n >> 1) & 1), abort_flag, status);
            __syncwarp();
            smc_tc_fence_after();
            const uint32_t src = tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(buf * BN);
            for (int c = 0; c < BN; c += 32) {
                uint32_t r[2][16];
                smc_tc_ld16(src + (uint32_t)c, r[0]);
                smc_tc_ld16(src + (uint32_t)c + 16u, r[1]);
                smc_tc_wait_ld();
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int nc = n0 + c + 16 * h;
                    if (m >= M || nc >= N) continue;
                    float v[16];
#pragma unroll
                    for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[h][i]);
                    constexpr bool PAIRS = EPI == EPI_SILU_PAIRS || EPI == EPI_GELU_PAIRS;
                    if (PAIRS) {
                        float f[8];
                        if (o.y_bf16) {
#pragma unroll
                            for (int i = 0; i < 8; ++i) f[i] = act_pair_fast<EPI == EPI_GELU_PAIRS>(v[2 * i], v[2 * i + 1]);
                        } else {
#pragma unroll
                            for (int i = 0; i < 8; ++i) f[i] = act_pair(EPI == EPI_GELU_PAIRS ? 2 : 1, v[2 * i], v[2 * i + 1]);
                        }
                        const int c2 = nc >> 1;
                        if (o.y_bf16 && nc + 16 <= N && (o.ldy & 7) == 0) {
                            __nv_bfloat162 p[4];
#pragma unroll
                            for (int i = 0; i < 4; ++i) p[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
                            *reinterpret_cast<uint4 *>(static_cast<bf16 *>(o.y) + (size_t)m * o.ldy + c2) = *reinterpret_cast<uint4 *>(p);
                        } else {
#pragma unroll
                            for (int i = 0; i < 8; ++i)
                                if (nc + 2 * i + 1 < N) {
                                    if (o.y_bf16) static_cast<bf16 *>(o.y)[(size_t)m * o.ldy + c2 + i] = __float2bfloat16_rn(f[i]);
                                    else static_cast<float *>(o.y)[(size_t)m * o.ldy + c2 + i] = f[i];
                                }
                        }
                    } else if (nc + 16 <= N && (o.split == 0 || nc + 16 <= o.split) && (o.ldy & 7) == 0) {
                        if (EPI == EPI_FINISH) {
                            if (o.bias) {
#pragma unroll
                                for (int i = 0; i < 4; ++i) {
                                    const float4 b = __ldg(reinterpret_cast<const float4 *>(o.bias + nc) + i);
                                    v[4 * i] += b.x, v[4 * i + 1] += b.y, v[4 * i + 2] += b.z, v[4 * i + 3] += b.w;
                                }
                            }
                            if (nc >= o.silu_from && nc + 16 <= o.silu_to && o.y_bf16) {
#pragma unroll
                                for (int i = 0; i < 16; ++i) v[i] = silu_for<bf16>(v[i]);
                            } else if (nc < o.silu_to && nc + 16 > o.silu_from) {
#pragma unroll
                                for (int i = 0; i < 16; ++i) v[i] = nc + i >= o.silu_from && nc + i < o.silu_to ? silu(v[i]) : v[i];
                            }
                            if (o.softcap > 0.f) {
#pragma unroll
                                for (int i = 0; i < 16; ++i) v[i] = o.softcap * tanhf(__fdiv_rn(v[i], o.softcap));
                            }
                        }
                        if (o.y_bf16) {
                            __nv_bfloat162 p[8];
#pragma unroll
                            for (int i = 0; i < 8; ++i) p[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
                            uint4 *dst = reinterpret_cast<uint4 *>(static_cast<bf16 *>(o.y) + (size_t)m * o.ldy + nc);
                            dst[0] = reinterpret_cast<uint4 *>(p)[0], dst[1] = reinterpret_cast<uint4 *>(p)[1];
                        } else {
                            float4 *dst = reinterpret_cast<float4 *>(static_cast<float *>(o.y) + (size_t)m * o.ldy + nc);
#pragma unroll
                            for (int i = 0; i < 4; ++i) {
                                if (o.accumulate) add4(reinterpret_cast<float *>(dst + i), v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
                                else dst[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
                            }
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (nc + i < N) put(o, m, nc + i, v[i]);
                    }
                }
                __syncwarp();  // the accumulator reads are warp-wide: lanes without a token rejoin here
            }
            smc_tc_fence_before();
            __syncwarp();
            if (lane == 0) smc_mbar_arrive(acc_empty(buf));
        }
    }
    smc_tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        __syncwarp();
        smc_tc_dealloc(tmem, S::COLS);
    }
}

typedef CUresult (*encode_fn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                              const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

encode_fn tensor_map_encoder()
{
    static encode_fn fn = [] {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) p = nullptr;
        return reinterpret_cast<encode_fn>(p);
    }();
    return fn;
}

// [rows, cols] bfloat16 with row stride ld elements, boxes of box_rows x 64
bool make_map(CUtensorMap *map, const void *base, uint64_t cols, uint64_t rows, uint64_t ld, uint32_t box_rows)
{
    encode_fn fn = tensor_map_encoder();
    if (!fn) return false;
    const cuuint64_t dims[2] = {cols, rows}, strides[1] = {ld * 2};
    const cuuint32_t box[2] = {TC_K, box_rows}, es[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN, int EPI>
int launch_tc(smc_ctx *ctx, const bf16 *x, int ldx, const bf16 *w, int M, int N, int K, const smc_dense_out &o, cudaStream_t s)
{
    using S = TcShape<BN>;
    CUtensorMap mx, mw;
    if (!make_map(&mx, x, K, M, ldx, TC_M) || !make_map(&mw, w, K, N, K, BN)) return smc_fail(ctx, SMC_E_CUDA, "dense matmul: tensor map encoding failed");
    static bool attr_set = false;
    if (!attr_set) {
        SMC_CUDA(ctx, cudaFuncSetAttribute(dense_tc_kernel<BN, EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::SMEM));
        attr_set = true;
    }
    const int tiles = ((M + TC_M - 1) / TC_M) * ((N + BN - 1) / BN);
    smc_launch_dep(ctx->use_pdl, dense_tc_kernel<BN, EPI>, dim3(tiles < ctx->sm_count ? tiles : ctx->sm_count), dim3(192), S::SMEM, s, mx, mw, M, N, K, o,
                   ctx->d_status);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

void launch_skinny(smc_ctx *ctx, const bf16 *x, int ldx, int x_group, const bf16 *w, int groups, int N, int K, int M, const smc_dense_out &o, cudaStream_t s)
{
    const int nt = M <= 8 ? 1 : (M <= 16 ? 2 : 4), my = (M + nt * 8 - 1) / (nt * 8);
    const bool half = (long long)((N + 15) / 16) * my * groups < 2 * ctx->sm_count;  // fewer than two CTAs per SM
    const dim3 grid(half ? (N + 7) / 8 : (N + 15) / 16, my, groups);
    auto go = [&](auto kernel) { smc_launch_dep(ctx->use_pdl, kernel, grid, dim3(256), 0, s, w, x, ldx, M, N, K, o, x_group, NormedRow{}); };
    const bool deep = K >= 2048;  // eight chunks and more per warp
    if (nt == 1 && deep) half ? go(dense_skinny_kernel<1, 8, true>) : go(dense_skinny_kernel<1, 8, false>);
    else if (nt == 1) half ? go(dense_skinny_kernel<1, 4, true>) : go(dense_skinny_kernel<1, 4, false>);
    else if (nt == 2) half ? go(dense_skinny_kernel<2, 4, true>) : go(dense_skinny_kernel<2, 4, false>);
    else half ? go(dense_skinny_kernel<4, 4, true>) : go(dense_skinny_kernel<4, 4, false>);
}

// one fp32 row, layer-normed on the way
template <int KV, int U>
void launch_skinny_normed(smc_ctx *ctx, const NormedRow &row, const bf16 *w, int N, int K, const smc_dense_out &o, cudaStream_t s)
{
    const bool half = (N + 15) / 16 < 2 * ctx->sm_count;
    auto go = [&](auto kernel) {
        smc_launch_dep(ctx->use_pdl, kernel, dim3(half ? (N + 7) / 8 : (N + 15) / 16), dim3(256), 0, s, w, (const bf16 *)nullptr, 0, 1, N, K, o, 0, row);
    };
    half ? go(dense_skinny_kernel<1, U, true, KV>) : go(dense_skinny_kernel<1, U, false, KV>);
}

__global__ void __launch_bounds__(256) round_bf16_kernel(const float *__restrict__ x, bf16 *__restrict__ y, long long n)
{
    smc_grid_dep_sync();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i < n) y[i] = __float2bfloat16_rn(x[i]);
}

}  // namespace

int smc_launch_round_bf16(smc_ctx *ctx, const float *x, void *y, long long n, cudaStream_t s)
{
    smc_launch_dep(ctx->use_pdl, round_bf16_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, x, static_cast<bf16 *>(y), n);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

int smc_launch_dense_rows(smc_ctx *ctx, const void *x, int x_bf16, int ldx, const smc_weight *wt, int row0, int N, int M, const smc_dense_out &o,
                          cudaStream_t s)
{
    if (wt->dtype != SMC_BF16) return smc_fail(ctx, SMC_E_UNSUPPORTED, "dense matmul: the weight is not bfloat16");
    const int K = wt->K;
    const bf16 *w = reinterpret_cast<const bf16 *>(wt->d_raw) + (size_t)row0 * K;
    auto aligned = [](const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = x_bf16 && K % 8 == 0 && ldx % 8 == 0 && aligned(x) && aligned(w);
    if (vec) {
        const bf16 *xb = static_cast<const bf16 *>(x);
        if (M > 32 && aligned(o.y) && aligned(o.bias)) {
            // rounds of tiles over the device: a wide tile takes less than twice as long as a narrow one
            const long long mt = (M + TC_M - 1) / TC_M, sms = ctx->sm_count;
            const long long wide = 2 * ((mt * ((N + 255) / 256) + sms - 1) / sms), narrow = (mt * ((N + 127) / 128) + sms - 1) / sms;
            auto tc = [&](auto epi) {
                constexpr int E = decltype(epi)::value;
                return 5 * wide <= 6 * narrow ? launch_tc<256, E>(ctx, xb, ldx, w, M, N, K, o, s) : launch_tc<128, E>(ctx, xb, ldx, w, M, N, K, o, s);
            };
            if (o.woven == 2) return tc(std::integral_constant<int, EPI_GELU_PAIRS>());
            if (o.woven) return tc(std::integral_constant<int, EPI_SILU_PAIRS>());
            if (o.bias || o.silu_to > o.silu_from || o.softcap > 0.f) return tc(std::integral_constant<int, EPI_FINISH>());
            return tc(std::integral_constant<int, EPI_STORE>());
        }
        launch_skinny(ctx, xb, ldx, 0, w, 1, N, K, M, o, s);
        SMC_LAUNCH_CHECK(ctx);
        return SMC_OK;
    }
    auto go = [&](auto *xp) {
        using TX = std::remove_const_t<std::remove_pointer_t<decltype(xp)>>;
        if (M <= 16) {
            const int warps = o.woven ? N / 2 : N;
            smc_launch_dep(ctx->use_pdl, dense_rows_kernel<TX>, dim3((warps + 7) / 8, (M + 7) / 8), dim3(256), 0, s, w, xp, ldx, M, N, K, o);
        } else {
            smc_launch_dep(ctx->use_pdl, dense_tile_kernel<TX>, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, s, w, xp, ldx, M, N, K, o);
        }
    };
    if (x_bf16) go(static_cast<const bf16 *>(x));
    else go(static_cast<const float *>(x));
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

int smc_launch_dense_grouped(smc_ctx *ctx, const void *x, int ldx, int x_group, const void *w, int groups, int N, int K, int M, const smc_dense_out &o,
                             cudaStream_t s)
{
    if (K % 8 || ldx % 8 || x_group % 8 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(w) & 15))
        return smc_fail(ctx, SMC_E_UNSUPPORTED, "grouped dense matmul: rows must start on 16-byte boundaries");
    const bf16 *xb = static_cast<const bf16 *>(x), *wb = static_cast<const bf16 *>(w);
    launch_skinny(ctx, xb, ldx, x_group, wb, groups, N, K, M, o, s);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

int smc_launch_dense(smc_ctx *ctx, const void *x, int x_bf16, int ldx, const smc_weight *w, int M, const smc_dense_out &o, cudaStream_t s)
{
    return smc_launch_dense_rows(ctx, x, x_bf16, ldx, w, 0, w->N, M, o, s);
}

int smc_launch_dense_layernorm(smc_ctx *ctx, const float *x, const float *norm, float eps, void *scratch, int scratch_bf16, const smc_weight *wt, int M,
                               const smc_dense_out &o, cudaStream_t s)
{
    const int K = wt->K;
    auto aligned = [](const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    // worth it while one wave of CTAs covers the matrix: the CTAs of a later wave would norm the row again with nothing to hide it
    if (M == 1 && scratch_bf16 && wt->dtype == SMC_BF16 && K % 8 == 0 && K <= 1024 && (wt->N + 15) / 16 <= 3 * ctx->sm_count && aligned(x) && aligned(norm) && aligned(wt->d_raw)) {
        const NormedRow row{x, norm, eps};
        const bf16 *w = reinterpret_cast<const bf16 *>(wt->d_raw);
        launch_skinny_normed<1, 4>(ctx, row, w, wt->N, K, o, s);
        SMC_LAUNCH_CHECK(ctx);
        return SMC_OK;
    }
    int rc = smc_launch_layernorm(ctx, x, nullptr, 0, M, norm, scratch, scratch_bf16, K, eps, s);
    return rc ? rc : smc_launch_dense(ctx, scratch, scratch_bf16, K, wt, M, o, s);
}
