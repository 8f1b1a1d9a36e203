// State-space (Mamba-2) sequence mixing between its two projections:
//   x | B | C pass a causal convolution per channel and SiLU;  dt = softplus(dt_raw + bias)
//   S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t        per head, S [state, vdim]
//   o = RMSNorm in parts(y * SiLU(z)) * w
// Two forms of the recurrence: token after token (ssm_scan_kernel: decoding, short portions, fp32, odd sizes), and chunks of
// 64 tokens whose inner sums are matrix products on the tensor cores (ssm_chunk_kernel).
// dt, decays, S and y are fp32.  A sequence's state is S and the inputs of the convolution's last taps (position p in row
// p % taps of its ring).
#include <type_traits>

#include "smc_mma.cuh"

namespace {

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------ convolution
// A thread walks CR rows of V neighbouring channels, the last taps inputs in registers (TAPS = 0: taps read again for every
// row, any number of them).  Inputs before the portion come from the ring; those before position 0 are zero.  One row per
// sequence (decoding): the same launch stores the row's input, whose ring place nobody reads any more.
constexpr int CR = 16;
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const T *__restrict__ zx, int ld, int inner, T *__restrict__ out, T *__restrict__ ring, smc_rows rw,
                                                       const float *__restrict__ w, const float *__restrict__ b, int ch, int ntaps)
{
    const int taps = TAPS ? TAPS : ntaps;
    const int c = (blockIdx.x * 128 + threadIdx.x) * V;
    const bool seq = rw.seq0 >= 0;
    float wc[V][TAPS ? TAPS : 1], bias[V];
    if (c < ch) {
#pragma unroll
        for (int i = 0; i < V; ++i) {
            bias[i] = b[c + i];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) wc[i][j] = w[(size_t)(c + i) * taps + j];
        }
    }
    smc_grid_dep_sync();
    if (c >= ch) return;
    const int r0 = blockIdx.y * (seq ? CR : 1), r1 = min(rw.n, r0 + (seq ? CR : 1)), first = seq ? 0 : r0;  // rows before `first` are other sequences'
    const int slot = seq ? rw.seq0 : r0, p0 = rw.pos[slot] - (seq ? 0 : r0);                                 // row r is at position p0 + r
    T *rg = ring + (size_t)slot * taps * ch + c;
    auto input = [&](int r, float (&v)[V]) {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = 0.f;
        if (p0 + r < 0) return;
        if (r >= first) load_v<T, V>(zx + (size_t)r * ld + inner + c, v);
        else load_v<T, V>(rg + (size_t)((p0 + r) % taps) * ch, v);
    };
    if (TAPS) {
        float hist[TAPS ? TAPS : 1][V];  // hist[j]: input of row r - taps + 1 + j
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) input(r0 - TAPS + 1 + j, hist[j + 1]);
        for (int rb = r0; rb < r1; rb += 8) {
            typename Pack<T, V>::type raw[8];
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (rb + k < r1) raw[k] = *reinterpret_cast<const typename Pack<T, V>::type *>(zx + (size_t)(rb + k) * ld + inner + c);
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                if (rb + k >= r1) break;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                    for (int i = 0; i < V; ++i) hist[j][i] = hist[j + 1][i];
                float v[V];
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    hist[TAPS - 1][i] = to_f(reinterpret_cast<const T *>(&raw[k])[i]);
                    v[i] = bias[i];
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) v[i] = fmaf(wc[i][j], hist[j][i], v[i]);
                    v[i] = silu_for<T>(v[i]);
                }
                store_v<T, V>(out + (size_t)(rb + k) * ch + c, v);
            }
        }
    } else {
        for (int r = r0; r < r1; ++r) {
            float v[V], x[V];
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = bias[i];
            for (int j = 0; j < taps; ++j) {
                input(r - taps + 1 + j, x);
#pragma unroll
                for (int i = 0; i < V; ++i) v[i] = fmaf(w[(size_t)(c + i) * taps + j], x[i], v[i]);
            }
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = silu_for<T>(v[i]);
            store_v<T, V>(out + (size_t)r * ch + c, v);
        }
    }
    if (!seq || rw.n == 1)
        *reinterpret_cast<typename Pack<T, V>::type *>(rg + (size_t)((p0 + r0) % taps) * ch) =
            *reinterpret_cast<const typename Pack<T, V>::type *>(zx + (size_t)r0 * ld + inner + c);
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
constexpr int CQ = 64, CP = 32, CTH = 512;
struct ChunkSmem {  // byte offsets; rows are padded to an odd number of 16-byte units
    int ldn, cb, x, m, xw, st, f, total;
};
__host__ __device__ constexpr ChunkSmem chunk_smem(int N)
{
    ChunkSmem o{};
    const int n16 = (N + 15) & ~15;
    o.ldn = (n16 + 8) * 2;
    o.cb = 0;                                   // two buffers of C [64][N] then B [64][N]
    o.x = o.cb + 4 * CQ * o.ldn;                // two buffers of x [64][32]
    o.m = o.x + 2 * CQ * 80;                    // weights hi, lo [64][64]
    o.xw = o.m + 2 * CQ * 144;                  // scaled x hi, lo [64][32]
    o.st = o.xw + 2 * CQ * 80;                  // state hi, lo [32][N]
    o.f = o.st + 2 * CP * o.ldn + 32;           // two buffers of dt, c, 2^c, 2^(c_end - c) dt [64] fp32 each, then 2^c_end
    o.total = o.f + 2 * (4 * CQ + 4) * 4;
    return o;
}

// 16 warps: token tile warp % 4 against a quarter of the other side.
template <int NTW, int NC>  // state tiles of 8 columns per warp (eight warps across N); N if known, 0: any up to 64 NTW
__global__ void __launch_bounds__(CTH) ssm_chunk_kernel(const bf16 *__restrict__ xbc, const float *__restrict__ dt_raw, float *__restrict__ y,
                                                        float *__restrict__ state, smc_rows rw, const float *__restrict__ dt_bias,
                                                        const float *__restrict__ a_log, const float *__restrict__ d_skip, int heads, int P, int N_,
                                                        int groups)
{
    const int N = NC ? NC : N_;
    extern __shared__ __align__(16) uint8_t csm[];
    const ChunkSmem L = chunk_smem(N);
    const uint32_t sb = (uint32_t)__cvta_generic_to_shared(csm);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int h = blockIdx.x, p0 = blockIdx.y * CP, grp = h / (heads / groups), T = rw.n;
    const int inner = heads * P, ch = inner + 2 * groups * N, n16 = (N + 15) & ~15, ksteps = n16 / 16;
    for (int e = threadIdx.x; e < L.total / 16; e += CTH) reinterpret_cast<uint4 *>(csm)[e] = make_uint4(0u, 0u, 0u, 0u);
    smc_grid_dep_sync();
    __syncthreads();
    const bool fresh = rw.pos[rw.seq0] == 0;
    float *st = state + ((size_t)rw.seq0 * heads + h) * P * N;
    const float D = d_skip[h], bias = dt_bias[h];
    const double A2 = -(double)expf(a_log[h]) * 1.4426950408889634;  // log decays are kept as powers of two
    const int cn = N / 8, cx = min(CP, P - p0) / 8, per = 2 * cn + cx;
    const int ft0 = threadIdx.x / per, fc0 = threadIdx.x % per, fts = CTH / per, fcs = CTH % per;  // the copies' (token, piece), stepped without divisions
    auto fetch = [&](int t0, int buf) {
        for (int t = ft0, c = fc0; t < CQ; t += fts, c += fcs) {
            if (c >= per) {
                c -= per;
                if (++t >= CQ) break;
            }
            const bool in = t0 + t < T;
            const bf16 *src = xbc + (size_t)(in ? t0 + t : T - 1) * ch;
            if (c < cn) cp16(sb + L.cb + (uint32_t)((2 * buf * CQ + t) * L.ldn + 16 * c), src + inner + (groups + grp) * N + 8 * c, in);
            else if (c < 2 * cn) cp16(sb + L.cb + (uint32_t)(((2 * buf + 1) * CQ + t) * L.ldn + 16 * (c - cn)), src + inner + grp * N + 8 * (c - cn), in);
            else cp16(sb + L.x + (uint32_t)((buf * CQ + t) * 80 + 16 * (c - 2 * cn)), src + h * P + p0 + 8 * (c - 2 * cn), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // step sizes and running log decays of a chunk by one warp, two tokens per lane; past the end: no input, no decay
    float raw0 = 0.f, raw1 = 0.f;
    auto load_dt = [&](int t0) {
        const int t = t0 + 2 * lane;
        raw0 = t < T ? dt_raw[(size_t)t * heads + h] : 0.f, raw1 = t + 1 < T ? dt_raw[(size_t)(t + 1) * heads + h] : 0.f;
    };
    auto prepare = [&](int t0, int buf) {
        float *f = reinterpret_cast<float *>(csm + L.f) + buf * (4 * CQ + 4);
        const int t = t0 + 2 * lane;
        const float d0 = t < T ? softplus(raw0 + bias) : 0.f, d1 = t + 1 < T ? softplus(raw1 + bias) : 0.f;
        const double a1 = A2 * d1;
        double sum = A2 * d0 + a1;
        for (int d = 1; d < 32; d <<= 1) {
            const double v = __shfl_up_sync(0xffffffffu, sum, d);
            if (lane >= d) sum += v;
        }
        const double end = __shfl_sync(0xffffffffu, sum, 31);
        const float c0 = (float)(sum - a1), c1 = (float)sum;
        *reinterpret_cast<float2 *>(f + 2 * lane) = make_float2(d0, d1);
        *reinterpret_cast<float2 *>(f + CQ + 2 * lane) = make_float2(c0, c1);
        *reinterpret_cast<float2 *>(f + 2 * CQ + 2 * lane) = make_float2(ex2(c0), ex2(c1));
        *reinterpret_cast<float2 *>(f + 3 * CQ + 2 * lane) = make_float2(ex2((float)(end - (sum - a1))) * d0, ex2((float)(end - sum)) * d1);
        if (lane == 0) f[4 * CQ] = ex2((float)end);
    };
    fetch(0, 0);
    if (warp == 0) load_dt(0), prepare(0, 0);
    // state accumulators: rows p (two tiles of 16), columns n (an eighth each)
    const int sm_m = warp & 1, sm_n = warp >> 1;
    float S[NTW][4];
    const int nt_per = (n16 / 8 + 7) / 8;
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
    const int mt = warp & 3, nq = warp >> 2;
    int buf = 0;
    for (int t0 = 0; t0 < T; t0 += CQ, buf ^= 1) {
        const bool more = t0 + CQ < T;
        if (more) {
            fetch(t0 + CQ, buf ^ 1);
            if (warp == 0) load_dt(t0 + CQ);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float *s_dt = reinterpret_cast<const float *>(csm + L.f) + buf * (4 * CQ + 4), *s_c = s_dt + CQ, *s_ec = s_c + CQ, *s_w = s_ec + CQ;
        const uint32_t cC = sb + L.cb + (uint32_t)(2 * buf * CQ * L.ldn), cB = cC + (uint32_t)(CQ * L.ldn), cX = sb + L.x + (uint32_t)(buf * CQ * 80);
        // ---- C_t . B_s for 16 tokens x 16 sources, and S^T C for 16 tokens x 8 value columns
        float G[2][4], Y[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
        const bool any = nq <= mt;  // else every source lies after every token
#pragma unroll
        for (int k = 0; k < ksteps; k += 2) {
            uint32_t sh[4], sl[4];  // eight state rows for two k-steps (of an odd last pair only the first half is used)
            ldsm4(sb + L.st + (uint32_t)((8 * nq + (lane & 7)) * L.ldn + 32 * k + 16 * (lane >> 3)), sh);
            ldsm4(sb + L.st + (uint32_t)((CP + 8 * nq + (lane & 7)) * L.ldn + 32 * k + 16 * (lane >> 3)), sl);
#pragma unroll
            for (int j = 0; j < 2; ++j)
                if (k + j < ksteps) {
                    uint32_t a[4];
                    ldsm4(cC + (uint32_t)((16 * mt + la) * L.ldn + 32 * (k + j) + lah), a);
                    if (any) {
                        uint32_t b[4];
                        ldsm4(cB + (uint32_t)((16 * nq + lb) * L.ldn + 32 * (k + j) + lbh), b);
                        mma_bf16(G[0], a, b[0], b[1]);
                        mma_bf16(G[1], a, b[2], b[3]);
                    }
                    mma_bf16(Y[0], a, sl[2 * j], sl[2 * j + 1]);
                    mma_bf16(Y[1], a, sh[2 * j], sh[2 * j + 1]);
                }
        }
        const int ta = 16 * mt + g, tb = ta + 8;
        if (any) {
            const float ca = s_c[ta], cb = s_c[tb];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int s = 16 * nq + 8 * i + 2 * tg;
                const float2 cs = *reinterpret_cast<const float2 *>(s_c + s), ds = *reinterpret_cast<const float2 *>(s_dt + s);
                // (a source after the token would have a growing factor: its exponent is clamped and its weight zeroed)
                const float w0 = s <= ta ? G[i][0] * (ex2(fminf(ca - cs.x, 0.f)) * ds.x) : 0.f, w1 = s + 1 <= ta ? G[i][1] * (ex2(fminf(ca - cs.y, 0.f)) * ds.y) : 0.f;
                const float w2 = s <= tb ? G[i][2] * (ex2(fminf(cb - cs.x, 0.f)) * ds.x) : 0.f, w3 = s + 1 <= tb ? G[i][3] * (ex2(fminf(cb - cs.y, 0.f)) * ds.y) : 0.f;
                uint32_t hi, lo;
                uint8_t *d = csm + L.m + ta * 144 + 2 * s;
                split2(w0, w1, hi, lo);
                *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CQ * 144) = lo;
                split2(w2, w3, hi, lo);
                d += 8 * 144;
                *reinterpret_cast<uint32_t *>(d) = hi, *reinterpret_cast<uint32_t *>(d + CQ * 144) = lo;
            }
        }
        const float ea = s_ec[ta], eb = s_ec[tb];
        Y[0][0] = (Y[0][0] + Y[1][0]) * ea, Y[0][1] = (Y[0][1] + Y[1][1]) * ea, Y[0][2] = (Y[0][2] + Y[1][2]) * eb, Y[0][3] = (Y[0][3] + Y[1][3]) * eb;
        Y[1][0] = Y[1][1] = Y[1][2] = Y[1][3] = 0.f;
        // ---- x scaled for the state update
#pragma unroll
        for (int e = threadIdx.x; e < CQ * CP / 2; e += CTH) {
            const int t = e >> 4, c = (e & 15) * 2;
            const float f = s_w[t];
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162 *>(csm + L.x + (buf * CQ + t) * 80 + 2 * c);
            uint32_t hi, lo;
            split2(__bfloat162float(v.x) * f, __bfloat162float(v.y) * f, hi, lo);
            *reinterpret_cast<uint32_t *>(csm + L.xw + t * 80 + 2 * c) = hi, *reinterpret_cast<uint32_t *>(csm + L.xw + (CQ + t) * 80 + 2 * c) = lo;
        }
        __syncthreads();
        // ---- y: weights times x, sources up to the tile's last token (weights past it were never written: stay below)
#pragma unroll
        for (int k = 0; k < CQ / 16; k += 2) {
            if (k > mt) break;
            uint32_t b[4];  // eight value columns for 32 sources
            ldsm4t(cX + (uint32_t)((16 * k + lane) * 80 + 16 * nq), b);
#pragma unroll
            for (int j = 0; j < 2; ++j)
                if (k + j <= mt) {
                    uint32_t ah[4], al[4];
                    ldsm4(sb + L.m + (uint32_t)((16 * mt + la) * 144 + 32 * (k + j) + lah), ah);
                    ldsm4(sb + L.m + (uint32_t)((CQ + 16 * mt + la) * 144 + 32 * (k + j) + lah), al);
                    mma_bf16(Y[1], al, b[2 * j], b[2 * j + 1]);
                    mma_bf16(Y[0], ah, b[2 * j], b[2 * j + 1]);
                }
        }
        {
            const int c = 8 * nq + 2 * tg;
            if (p0 + c < P) {
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int t = ta + 8 * j;
                    if (t0 + t >= T) continue;
                    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162 *>(csm + L.x + (buf * CQ + t) * 80 + 2 * c);
                    *reinterpret_cast<float2 *>(y + (size_t)(t0 + t) * inner + h * P + p0 + c) =
                        make_float2(fmaf(D, __bfloat162float(v.x), Y[0][2 * j] + Y[1][2 * j]), fmaf(D, __bfloat162float(v.y), Y[0][2 * j + 1] + Y[1][2 * j + 1]));
                }
            }
        }
        // ---- state
        const float dec = s_dt[4 * CQ];
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
                // two tiles; where the second lies past the row's end the first is read twice, where it is another warp's it is not used
                ldsm4t(cB + (uint32_t)((16 * k + la) * L.ldn + 16 * nt + (nt * 8 + 8 < n16 ? lah : 0)), b);
                mma_bf16(S[i], al, b[0], b[1]), mma_bf16(S[i], ah, b[0], b[1]);
                if (i + 1 < nt_per) mma_bf16(S[i + 1], al, b[2], b[3]), mma_bf16(S[i + 1], ah, b[2], b[3]);
            }
        }
        if (warp == 0 && more) prepare(t0 + CQ, buf ^ 1);  // this warp has the least of the triangle above
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
template <typename T, int V>
__global__ void __launch_bounds__(128) ssm_gate_norm_kernel(const float *__restrict__ y, const T *__restrict__ zx, int ld, const float *__restrict__ w,
                                                            T *__restrict__ o, int inner, int parts, float eps)
{
    extern __shared__ __align__(16) float sv[];
    __shared__ float red[4];
    smc_grid_dep_sync();
    const int n = inner / parts, r = blockIdx.x, base = blockIdx.y * n;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < n; i += 128 * V) {
        float a[V], z[V];
        load_v<float, V>(y + (size_t)r * inner + base + i, a);
        load_v<T, V>(zx + (size_t)r * ld + base + i, z);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] *= silu_for<T>(z[j]), ss = fmaf(a[j], a[j], ss);
        store_v<float, V>(sv + i, a);
    }
    ss = smc_group_sum<32>(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = (red[0] + red[1]) + (red[2] + red[3]);
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)n) + eps));
    for (int i = threadIdx.x * V; i < n; i += 128 * V) {
        float a[V], g[V];
        load_v<float, V>(sv + i, a);
        load_v<float, V>(w + base + i, g);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = (a[j] * inv) * g[j];
        store_v<T, V>(o + (size_t)r * inner + base + i, a);
    }
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
        smc_launch_dep(ctx->use_pdl, kernel, dim3(d.heads, (d.vdim + CP - 1) / CP), dim3(CTH), (size_t)L.total, s, (const bf16 *)b.xbc, b.dt_raw, b.y,
                       b.state, rw, dt_bias, a_log, d_skip, d.heads, d.vdim, d.state, d.groups);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    if (d.state == 128) return go(ssm_chunk_kernel<2, 128>);
    if (d.state == 64) return go(ssm_chunk_kernel<2, 64>);
    return d.state <= 128 ? go(ssm_chunk_kernel<2, 0>) : go(ssm_chunk_kernel<4, 0>);
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
    auto conv = [&](auto kernel, int v) {
        smc_launch_dep(ctx->use_pdl, kernel, dim3((ch / v + 127) / 128, seq ? (rw.n + CR - 1) / CR : rw.n), dim3(128), 0, s, static_cast<const T *>(b.zx),
                       b.ld, inner, static_cast<T *>(b.xbc), static_cast<T *>(b.conv_state), rw, conv_w, conv_b, ch, d.conv);
    };
    const bool four = inner % 4 == 0 && ch % 4 == 0 && b.ld % 4 == 0;
    if (d.conv == 4) four ? conv(ssm_conv_kernel<T, 4, 4>, 4) : conv(ssm_conv_kernel<T, 1, 4>, 1);
    else if (d.conv == 3) four ? conv(ssm_conv_kernel<T, 4, 3>, 4) : conv(ssm_conv_kernel<T, 1, 3>, 1);
    else if (d.conv == 2) four ? conv(ssm_conv_kernel<T, 4, 2>, 4) : conv(ssm_conv_kernel<T, 1, 2>, 1);
    else four ? conv(ssm_conv_kernel<T, 4, 0>, 4) : conv(ssm_conv_kernel<T, 1, 0>, 1);
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
    auto gate = [&](auto kernel) {
        if (nsm > 40 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)nsm);
        smc_launch_dep(ctx->use_pdl, kernel, dim3(rw.n, d.norm_groups), dim3(128), nsm, s, (const float *)b.y, static_cast<const T *>(b.zx), b.ld, norm,
                       static_cast<T *>(b.o), inner, d.norm_groups, d.eps);
    };
    if (inner / d.norm_groups % 4 == 0 && b.ld % 4 == 0) gate(ssm_gate_norm_kernel<T, 4>);
    else gate(ssm_gate_norm_kernel<T, 1>);
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
