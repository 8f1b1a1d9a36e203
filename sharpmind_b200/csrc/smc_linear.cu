// Linear attention with one fixed decay per head (lightning attention, retention) between its projections:
//   S_t = decay S_{t-1} + k_scale k_t v_t^T,   y_t = S_t^T q_t        per head, S [dim, vdim] fp32
//   o = norm in parts(y) * w * gate(g)
// with an optional rotation of the first elements of q and k.  Two forms of the recurrence:
//   token after token   linear_step_kernel: decoding, short portions, fp32, odd sizes
//   in chunks           (bfloat16 q, k, v) because the decay is fixed every chunk's own contribution is one matrix product
//                       (linear_state_kernel, all chunks at once), the states between chunks a running sum of those
//                       (linear_carry_kernel), and a chunk's outputs follow from the state before it and its own tokens
//                       (linear_out_kernel, all chunks at once).  fp32 factors (decayed weights, the state, the scaled
//                       values) enter the products as a pair hi + lo of bfloat16, i.e. with 16 bits; all sums are fp32.
#include <math.h>

#include <type_traits>

#include "smc_mma.cuh"

namespace {

// ------------------------------------------------------------------------------ token after token
// A CTA: one head of one sequence, 16 value columns; eight lanes share a column, a lane holding every eighth (group of four)
// of its states.  Steps are staged sixteen at a time, rotated and scaled on the way.  The state is requested before the
// wait for the predecessor (it was written by an earlier pass).
constexpr int SC = 16;
template <typename T, int NPL, bool VEC>
__global__ void __launch_bounds__(128) linear_step_kernel(const T *__restrict__ in, int ld, int col, float *__restrict__ y, float *state, smc_rows rw,
                                                          const float *__restrict__ decay, const float *__restrict__ cosT,
                                                          const float *__restrict__ sinT, int max_seq, int heads, int P, int N, int rd, float k_scale)
{
    extern __shared__ __align__(16) float sm[];
    const int h = blockIdx.x, c0 = blockIdx.y * 16, sub = threadIdx.x & 7, cc = threadIdx.x >> 3, p = c0 + cc;
    const bool seq = rw.seq0 >= 0;
    const int slot = seq ? rw.seq0 : (int)blockIdx.z, row0 = seq ? 0 : (int)blockIdx.z, T_ = seq ? rw.n : 1, cap = min(SC, T_);
    float *sq = sm, *sk = sq + cap * N, *sv = sk + cap * N;
    const int pos = rw.pos[slot];
    float *st = state + (((size_t)slot * heads + h) * P + min(p, P - 1)) * N;
    float S[NPL];
    auto at = [&](int j) { return VEC ? 4 * (sub + 8 * (j >> 2)) + (j & 3) : sub + 8 * j; };
    if (VEC) {
#pragma unroll
        for (int j = 0; j < NPL; j += 4) {
            const float4 v = pos != 0 && at(j) < N ? *reinterpret_cast<const float4 *>(st + at(j)) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[j] = v.x, S[j + 1] = v.y, S[j + 2] = v.z, S[j + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int j = 0; j < NPL; ++j) S[j] = pos != 0 && at(j) < N ? st[at(j)] : 0.f;
    }
    const float a = decay[h];
    smc_grid_dep_sync();
    const T *base = in + (size_t)row0 * ld + col;
    const int hN = heads * N, half = rd / 2;
    for (int t0 = 0; t0 < T_; t0 += SC) {
        const int nt = min(SC, T_ - t0);
        __syncthreads();
        for (int e = threadIdx.x; e < nt * N; e += 128) {
            const int t = e / N, i = e % N;
            const T *src = base + (size_t)(t0 + t) * ld + h * N;
            float q = to_f(src[i]), k = to_f(src[hN + i]);
            if (i < rd) {
                const int j = i < half ? i : i - half, other = i < half ? i + half : j;
                const size_t ti = (size_t)min(pos + t0 + t, max_seq - 1) * half + j;
                const float c = cosT[ti], s = i < half ? -sinT[ti] : sinT[ti];
                q = __fadd_rn(__fmul_rn(q, c), __fmul_rn(to_f(src[other]), s));
                k = __fadd_rn(__fmul_rn(k, c), __fmul_rn(to_f(src[hN + other]), s));
            }
            sq[e] = q, sk[e] = k * k_scale;
        }
        for (int e = threadIdx.x; e < nt * 16; e += 128)
            sv[e] = c0 + (e & 15) < P ? to_f(base[(size_t)(t0 + (e >> 4)) * ld + 2 * hN + h * P + c0 + (e & 15)]) : 0.f;
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = sv[t * 16 + cc];
            float acc = 0.f;
            if (VEC) {
#pragma unroll
                for (int j = 0; j < NPL; j += 4) {
                    if (at(j) >= N) continue;
                    const float4 k = *reinterpret_cast<const float4 *>(sk + t * N + at(j)), q = *reinterpret_cast<const float4 *>(sq + t * N + at(j));
                    S[j] = fmaf(k.x, v, a * S[j]), S[j + 1] = fmaf(k.y, v, a * S[j + 1]);
                    S[j + 2] = fmaf(k.z, v, a * S[j + 2]), S[j + 3] = fmaf(k.w, v, a * S[j + 3]);
                    acc = fmaf(S[j], q.x, acc), acc = fmaf(S[j + 1], q.y, acc), acc = fmaf(S[j + 2], q.z, acc), acc = fmaf(S[j + 3], q.w, acc);
                }
            } else {
#pragma unroll
                for (int j = 0; j < NPL; ++j) {
                    if (at(j) >= N) continue;
                    S[j] = fmaf(sk[t * N + at(j)], v, a * S[j]);
                    acc = fmaf(S[j], sq[t * N + at(j)], acc);
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (sub == 0 && p < P) y[((size_t)(row0 + t0 + t) * heads + h) * P + p] = acc;
        }
    }
    if (p >= P) return;
    if (VEC) {
#pragma unroll
        for (int j = 0; j < NPL; j += 4)
            if (at(j) < N) *reinterpret_cast<float4 *>(st + at(j)) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
    } else {
#pragma unroll
        for (int j = 0; j < NPL; ++j)
            if (at(j) < N) st[at(j)] = S[j];
    }
}

// ------------------------------------------------------------------------------ norm in parts, then gate
// o = y / rms(part) * w * gate(g) * out_scale; a warp (WARP) or a CTA per (row, part).  The gate's inputs were made by the
// kernel before the predecessor and are requested before the wait.
template <typename T> __device__ __forceinline__ float gate_of(int sigmoid, float g) { return sigmoid ? __fdiv_rn(1.0f, 1.0f + expf(-g)) : silu(g); }
template <> __device__ __forceinline__ float gate_of<bf16>(int sigmoid, float g) { return __fdividef(sigmoid ? 1.0f : g, 1.0f + __expf(-g)); }

template <typename T, int V, bool WARP>
__global__ void __launch_bounds__(256) norm_gate_kernel(const float *__restrict__ y, const T *__restrict__ g, int ld, const float *__restrict__ w,
                                                        T *__restrict__ o, int ldo, int rows, int inner, int parts, int sigmoid, float out_scale, float eps)
{
    constexpr int KEEP = 4;  // vectors a thread holds in registers; the rest is read again
    __shared__ float red[8];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n = inner / parts, step = (WARP ? 32 : 256) * V;
    const long long unit = WARP ? (long long)blockIdx.x * 8 + warp : blockIdx.x;
    const bool live = unit < (long long)rows * parts;
    const int r = live ? (int)(unit / parts) : 0, base = live ? (int)(unit % parts) * n : 0, i0 = (WARP ? lane : (int)threadIdx.x) * V;
    const float *yr = y + (size_t)r * inner + base;
    const T *gr = g + (size_t)r * ld + base;
    float gv[KEEP][V], yv[KEEP][V];
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (i0 + k * step < n) load_v<T, V>(gr + i0 + k * step, gv[k]);
    smc_grid_dep_sync();
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (i0 + k * step < n) {
            load_v<float, V>(yr + i0 + k * step, yv[k]);
#pragma unroll
            for (int j = 0; j < V; ++j) ss = fmaf(yv[k][j], yv[k][j], ss);
        }
    for (int i = i0 + KEEP * step; i < n; i += step) {
        float a[V];
        load_v<float, V>(yr + i, a);
#pragma unroll
        for (int j = 0; j < V; ++j) ss = fmaf(a[j], a[j], ss);
    }
    ss = smc_group_sum<32>(ss);
    if (!WARP) {
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = ((red[0] + red[1]) + (red[2] + red[3])) + ((red[4] + red[5]) + (red[6] + red[7]));
    }
    if (!live) return;
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)n) + eps));
    auto finish = [&](int i, float (&a)[V], float (&b)[V]) {
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = ((a[j] * inv) * (w ? w[base + i + j] : 1.0f)) * (gate_of<T>(sigmoid, b[j]) * out_scale);
        store_v<T, V>(o + (size_t)r * ldo + base + i, a);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (i0 + k * step < n) finish(i0 + k * step, yv[k], gv[k]);
    for (int i = i0 + KEEP * step; i < n; i += step) {
        float a[V], b[V];
        load_v<float, V>(yr + i, a);
        load_v<T, V>(gr + i, b);
        finish(i, a, b);
    }
}

// ------------------------------------------------------------------------------ chunks (bfloat16)
constexpr int CH = SMC_LINEAR_CHUNK, CTH = 256, PB = 64;  // tokens per chunk, threads, value columns per state CTA
__host__ __device__ constexpr int row_ld(int n) { return (((n + 15) & ~15) + 8) * 2; }  // bytes: an odd number of 16-byte units

// q and k [row, 2 heads, N] with the first rd elements rotated; a thread per V neighbouring pairs or unrotated elements
template <int V>
__global__ void __launch_bounds__(256) linear_rotate_kernel(const bf16 *__restrict__ in, int ld, int col, bf16 *__restrict__ qk, smc_rows rw,
                                                            const float *__restrict__ cosT, const float *__restrict__ sinT, int max_seq, int heads, int N,
                                                            int rd)
{
    smc_grid_dep_sync();
    const int half = rd / 2, units = (N - half) / V, e = blockIdx.x * 256 + threadIdx.x, r = blockIdx.y;
    if (e >= 2 * heads * units) return;
    const int u = e % units * V, h = e / units;
    const bf16 *src = in + (size_t)r * ld + col + (size_t)h * N;
    bf16 *dst = qk + ((size_t)r * 2 * heads + h) * N;
    float a[V], b[V];
    load_v<bf16, V>(src + half + u, b);
    if (u < half) {
        int slot, p;
        row_place(rw, r, slot, p);
        const size_t ti = (size_t)min(p, max_seq - 1) * half + u;
        float c[V], s[V];
        load_v<bf16, V>(src + u, a);
        load_v<float, V>(cosT + ti, c), load_v<float, V>(sinT + ti, s);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const float x = __fsub_rn(__fmul_rn(a[i], c[i]), __fmul_rn(b[i], s[i]));
            b[i] = __fadd_rn(__fmul_rn(b[i], c[i]), __fmul_rn(a[i], s[i])), a[i] = x;
        }
        store_v<bf16, V>(dst + u, a);
    }
    store_v<bf16, V>(dst + half + u, b);
}

// rows of a matrix -> shared memory, 16 bytes per copy, zeros from row `have` on
__device__ __forceinline__ void copy_rows(uint32_t dst, int ldd, const bf16 *src, size_t lds, int rows, int pieces, int have)
{
    const int lanes = pieces >= 16 ? 16 : (pieces >= 8 ? 8 : 4), c0 = threadIdx.x & (lanes - 1), j0 = threadIdx.x / lanes, js = CTH / lanes;
    for (int c = c0; c < pieces; c += lanes)
#pragma unroll 4
        for (int j = j0; j < rows; j += js) {
            const bool in = j < have;
            cp16(dst + (uint32_t)(j * ldd + 16 * c), in ? src + (size_t)j * lds + 8 * c : src, in);
        }
}

// What chunk z adds to a head's state: sum_s decay^(end - s) k_scale v_s k_s^T, 64 value columns x N per CTA.
template <int NT>  // tiles of 8 state columns per warp (two warps across N)
__global__ void __launch_bounds__(CTH) linear_state_kernel(const bf16 *__restrict__ k, size_t ldk, const bf16 *__restrict__ v, size_t ldv, float *__restrict__ part,
                                                           int T, const double *__restrict__ log2_decay, int heads, int P, int N, float k_scale)
{
    extern __shared__ __align__(16) uint8_t sm_raw[];
    constexpr int LV = (PB + 8) * 2;
    const int ldn = row_ld(N), lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int z = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PB, t0 = z * CH, len = min(CH, T - t0);
    const uint32_t sk = (uint32_t)__cvta_generic_to_shared(sm_raw), sv = sk + (uint32_t)(CH * ldn);
    uint8_t *vs = sm_raw + CH * ldn;
    const float l2d = (float)log2_decay[h];
    smc_grid_dep_sync();
    copy_rows(sk, ldn, k + (size_t)t0 * ldk + h * N, ldk, CH, N / 8, len);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const int cp = min(PB, P - p0) / 8;
    for (int e = threadIdx.x; e < CH * (PB / 8); e += CTH) {  // values times their decay, hi and lo
        const int t = e >> 3, c = e & 7;
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (t < len && c < cp) {
            const uint4 raw = *reinterpret_cast<const uint4 *>(v + (size_t)(t0 + t) * ldv + h * P + p0 + 8 * c);
            const bf16 *x = reinterpret_cast<const bf16 *>(&raw);
            const float f = k_scale * ex2((float)(len - 1 - t) * l2d);
            split2(to_f(x[0]) * f, to_f(x[1]) * f, hi.x, lo.x), split2(to_f(x[2]) * f, to_f(x[3]) * f, hi.y, lo.y);
            split2(to_f(x[4]) * f, to_f(x[5]) * f, hi.z, lo.z), split2(to_f(x[6]) * f, to_f(x[7]) * f, hi.w, lo.w);
        }
        *reinterpret_cast<uint4 *>(vs + t * LV + 16 * c) = hi, *reinterpret_cast<uint4 *>(vs + (CH + t) * LV + 16 * c) = lo;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int n16 = (N + 15) & ~15, mt = warp & 3, per = n16 / 16, nt0 = (warp >> 2) * per;
    float S[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < CH / 16; ++kk) {
        if (16 * kk >= len) break;
        uint32_t ah[4], al[4];
        const uint32_t off = (uint32_t)((16 * kk + (lane & 7) + 8 * (lane >> 4)) * LV + 32 * mt + 16 * ((lane >> 3) & 1));
        ldsm4t(sv + off, ah);
        ldsm4t(sv + (uint32_t)(CH * LV) + off, al);
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
            if (i >= per) continue;
            uint32_t b[4];  // two tiles; the second of an odd last pair is the other warp's, or padding: not used
            ldsm4t(sk + (uint32_t)((16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldn + 16 * (nt0 + i) + 16 * (lane >> 4)), b);
            mma_bf16(S[i], al, b[0], b[1]), mma_bf16(S[i], ah, b[0], b[1]);
            if (i + 1 < per) mma_bf16(S[i + 1], al, b[2], b[3]), mma_bf16(S[i + 1], ah, b[2], b[3]);
        }
    }
    float *dst = part + ((size_t)z * heads + h) * P * N;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int n = (nt0 + i) * 8 + 2 * tg, pa = p0 + 16 * mt + g;
        if (i >= per || n >= N) continue;
        if (pa < P) *reinterpret_cast<float2 *>(dst + (size_t)pa * N + n) = make_float2(S[i][0], S[i][1]);
        if (pa + 8 < P) *reinterpret_cast<float2 *>(dst + (size_t)(pa + 8) * N + n) = make_float2(S[i][2], S[i][3]);
    }
}

// The state before every chunk (bfloat16 hi and lo planes) and after the last; a thread per four elements.
__global__ void __launch_bounds__(256) linear_carry_kernel(const float4 *__restrict__ part, uint2 *__restrict__ start, float4 *__restrict__ state,
                                                           smc_rows rw, const double *__restrict__ log2_decay, int heads, int PN4)
{
    const int e = blockIdx.x * 256 + threadIdx.x, chunks = (rw.n + CH - 1) / CH;
    const bool live = e < heads * PN4;
    const int h = live ? e / PN4 : 0, i = live ? e % PN4 : 0;
    float4 *own = state + (size_t)rw.seq0 * heads * PN4 + (live ? e : 0);
    float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && rw.pos[rw.seq0] != 0) S = *own;
    const double l2 = log2_decay[h];
    const float f = exp2f((float)(CH * l2)), fl = exp2f((float)((rw.n - (chunks - 1) * CH) * l2));
    smc_grid_dep_sync();
    if (!live) return;
    constexpr int AHEAD = 8;
    for (int z0 = 0; z0 < chunks; z0 += AHEAD) {
        float4 u[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
            if (z0 + j < chunks) u[j] = part[((size_t)(z0 + j) * heads + h) * PN4 + i];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int z = z0 + j;
            if (z >= chunks) break;
            uint2 hi, lo;
            split2(S.x, S.y, hi.x, lo.x), split2(S.z, S.w, hi.y, lo.y);
            uint2 *dst = start + ((size_t)z * heads + h) * 2 * PN4 + i;
            dst[0] = hi, dst[PN4] = lo;
            const float d = z == chunks - 1 ? fl : f;
            S.x = fmaf(S.x, d, u[j].x), S.y = fmaf(S.y, d, u[j].y), S.z = fmaf(S.z, d, u[j].z), S.w = fmaf(S.w, d, u[j].w);
        }
    }
    *own = S;
}

// Outputs of chunk z of one head, up to 128 value columns; a warp per 16 tokens:
//   y_t = decay^(t+1) S^T q_t + sum_{s <= t} decay^(t-s) k_scale (q_t . k_s) v_s,  S the state before the chunk
// The second sum is attention without a softmax: weights go from the accumulators of the first product to the operands of the
// second in registers.  norm: the head is one part of the output norm, which is then taken here together with the gate.
struct OutArgs {
    const bf16 *q, *k, *v, *g;
    size_t ldq, ldk, ldv, ldg;
    const bf16 *start;
    float *y;
    bf16 *o;
    int ldo, norm, sigmoid;
    const float *w;
    float k_scale, out_scale, eps;
};
__host__ __device__ constexpr int out_smem(int P, int N)
{
    const int pb = P < 128 ? (P + 15) & ~15 : 128, planes = 2 * pb * row_ld(N), kv = CH * (row_ld(N) + row_ld(pb));
    return CH * row_ld(N) + (planes > kv ? planes : kv);
}
template <int VT>  // value tiles of 8 columns
__global__ void __launch_bounds__(CTH, 2) linear_out_kernel(OutArgs A, smc_rows rw, const double *__restrict__ log2_decay, int heads, int P, int N)
{
    extern __shared__ __align__(16) uint8_t sm_raw[];
    const int T = rw.n, ldn = row_ld(N), n16 = (N + 15) & ~15, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int z = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * 128, pn = min(128, P - p0), pb = (pn + 15) & ~15, ldp = row_ld(pb);
    const int t0 = z * CH, len = min(CH, T - t0);
    const uint32_t sq = (uint32_t)__cvta_generic_to_shared(sm_raw), s2 = sq + (uint32_t)(CH * ldn);
    const float l2d = (float)log2_decay[h];
    if (n16 != N) {  // padding of the contracted elements must be zero
        for (int e = threadIdx.x; e < out_smem(P, N) / 16; e += CTH) reinterpret_cast<uint4 *>(sm_raw)[e] = make_uint4(0u, 0u, 0u, 0u);
        __syncthreads();
    }
    smc_grid_dep_sync();
    const bool empty = z == 0 && rw.pos[rw.seq0] == 0;  // no state before the first token
    copy_rows(sq, ldn, A.q + (size_t)t0 * A.ldq + h * N, A.ldq, CH, N / 8, len);
    if (!empty) {
        const bf16 *src = A.start + (((size_t)z * heads + h) * 2 * P + p0) * N;
        copy_rows(s2, ldn, src, N, pb, N / 8, pn);
        copy_rows(s2 + (uint32_t)(pb * ldn), ldn, src + (size_t)P * N, N, pb, N / 8, pn);
    }
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();

    float Y[VT][4];
#pragma unroll
    for (int i = 0; i < VT; ++i) Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
    const int ta = 16 * warp + g, tb = ta + 8;
    const uint32_t a_off = sq + (uint32_t)((16 * warp + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldn + 16 * (lane >> 4));
    const uint32_t b_off = (uint32_t)(((lane & 7) + 8 * (lane >> 4)) * ldn + 16 * ((lane >> 3) & 1));
    if (!empty) {
#pragma unroll 2
        for (int ks = 0; ks < n16 / 16; ++ks) {
            uint32_t a[4];
            ldsm4(a_off + 32 * ks, a);
#pragma unroll
            for (int i = 0; i < VT / 2; ++i)
                if (16 * i < pb) {
                    uint32_t bh[4], bl[4];
                    ldsm4(s2 + b_off + (uint32_t)(16 * i * ldn + 32 * ks), bh);
                    ldsm4(s2 + b_off + (uint32_t)((pb + 16 * i) * ldn + 32 * ks), bl);
                    mma_bf16(Y[2 * i], a, bl[0], bl[1]), mma_bf16(Y[2 * i + 1], a, bl[2], bl[3]);
                    mma_bf16(Y[2 * i], a, bh[0], bh[1]), mma_bf16(Y[2 * i + 1], a, bh[2], bh[3]);
                }
        }
        const float ea = ex2((float)(ta + 1) * l2d), eb = ex2((float)(tb + 1) * l2d);
#pragma unroll
        for (int i = 0; i < VT; ++i) Y[i][0] *= ea, Y[i][1] *= ea, Y[i][2] *= eb, Y[i][3] *= eb;
        __syncthreads();  // the state planes make room for keys and values
    }
    const uint32_t sk = s2, sv = s2 + (uint32_t)(CH * ldn);
    copy_rows(sk, ldn, A.k + (size_t)t0 * A.ldk + h * N, A.ldk, CH, N / 8, len);
    copy_rows(sv, ldp, A.v + (size_t)t0 * A.ldv + h * P + p0, A.ldv, CH, pn / 8, len);
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int s0 = 0; s0 <= 16 * warp; s0 += 32) {  // 32 sources at a time, up to the warp's last token
        float G[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
        const bool second = s0 + 16 <= 16 * warp;
#pragma unroll 4
        for (int ks = 0; ks < n16 / 16; ++ks) {
            uint32_t a[4], b[4];
            ldsm4(a_off + 32 * ks, a);
            ldsm4(sk + b_off + (uint32_t)(s0 * ldn + 32 * ks), b);
            mma_bf16(G[0], a, b[0], b[1]), mma_bf16(G[1], a, b[2], b[3]);
            if (second) {
                ldsm4(sk + b_off + (uint32_t)((s0 + 16) * ldn + 32 * ks), b);
                mma_bf16(G[2], a, b[0], b[1]), mma_bf16(G[3], a, b[2], b[3]);
            }
        }
        uint32_t wh[2][4], wl[2][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int da = ta - (s0 + 8 * i + 2 * tg), db = da + 8;  // distances of the tile's first column; a source after the token has none
            const float f0 = da >= 0 ? G[i][0] * (A.k_scale * ex2((float)da * l2d)) : 0.f, f1 = da >= 1 ? G[i][1] * (A.k_scale * ex2((float)(da - 1) * l2d)) : 0.f;
            const float f2 = db >= 0 ? G[i][2] * (A.k_scale * ex2((float)db * l2d)) : 0.f, f3 = db >= 1 ? G[i][3] * (A.k_scale * ex2((float)(db - 1) * l2d)) : 0.f;
            split2(f0, f1, wh[i >> 1][(i & 1) * 2], wl[i >> 1][(i & 1) * 2]);
            split2(f2, f3, wh[i >> 1][(i & 1) * 2 + 1], wl[i >> 1][(i & 1) * 2 + 1]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            if (j == 1 && !second) break;
#pragma unroll
            for (int i = 0; i < VT / 2; ++i)
                if (16 * i < pb) {
                    uint32_t b[4];
                    ldsm4t(sv + (uint32_t)((s0 + 16 * j + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldp + 32 * i + 16 * (lane >> 4)), b);
                    mma_bf16(Y[2 * i], wl[j], b[0], b[1]), mma_bf16(Y[2 * i + 1], wl[j], b[2], b[3]);
                    mma_bf16(Y[2 * i], wh[j], b[0], b[1]), mma_bf16(Y[2 * i + 1], wh[j], b[2], b[3]);
                }
        }
    }
    if (!A.norm) {
#pragma unroll
        for (int i = 0; i < VT; ++i) {
            const int c = p0 + 8 * i + 2 * tg;
            if (c >= P) continue;
            if (ta < len) *reinterpret_cast<float2 *>(A.y + ((size_t)(t0 + ta) * heads + h) * P + c) = make_float2(Y[i][0], Y[i][1]);
            if (tb < len) *reinterpret_cast<float2 *>(A.y + ((size_t)(t0 + tb) * heads + h) * P + c) = make_float2(Y[i][2], Y[i][3]);
        }
        return;
    }
    float qa = 0.f, qb = 0.f;
#pragma unroll
    for (int i = 0; i < VT; ++i)
        if (8 * i < P) qa = fmaf(Y[i][0], Y[i][0], qa), qa = fmaf(Y[i][1], Y[i][1], qa), qb = fmaf(Y[i][2], Y[i][2], qb), qb = fmaf(Y[i][3], Y[i][3], qb);
    qa += __shfl_xor_sync(0xffffffffu, qa, 1), qa += __shfl_xor_sync(0xffffffffu, qa, 2);
    qb += __shfl_xor_sync(0xffffffffu, qb, 1), qb += __shfl_xor_sync(0xffffffffu, qb, 2);
    const float ia = __fdiv_rn(A.out_scale, sqrtf(__fdiv_rn(qa, (float)P) + A.eps)), ib = __fdiv_rn(A.out_scale, sqrtf(__fdiv_rn(qb, (float)P) + A.eps));
#pragma unroll
    for (int i = 0; i < VT; ++i) {
        const int c = 8 * i + 2 * tg;
        if (c >= P) continue;
        const float w0 = A.w ? A.w[h * P + c] : 1.f, w1 = A.w ? A.w[h * P + c + 1] : 1.f;
        auto put = [&](int t, float x, float y, float inv) {
            if (t >= len) return;
            const __nv_bfloat162 gg = *reinterpret_cast<const __nv_bfloat162 *>(A.g + (size_t)(t0 + t) * A.ldg + h * P + c);
            *reinterpret_cast<uint32_t *>(A.o + (size_t)(t0 + t) * A.ldo + h * P + c) =
                pack2(x * inv * w0 * gate_of<bf16>(A.sigmoid, __low2float(gg)), y * inv * w1 * gate_of<bf16>(A.sigmoid, __high2float(gg)));
        };
        put(ta, Y[i][0], Y[i][1], ia), put(tb, Y[i][2], Y[i][3], ib);
    }
}

// portions from this many rows on are taken in chunks
constexpr int CHUNK_ROWS = 32;

template <typename T>
int norm_gate(smc_ctx *ctx, const smc_linear_dims &d, const smc_linear_bufs &b, int rows, cudaStream_t s)
{
    const int inner = d.heads * d.vdim, n = inner / d.norm_parts, gc = b.col + 2 * d.heads * d.dim + inner;
    const T *g = static_cast<const T *>(b.in) + gc;
    auto go = [&](auto kernel, bool warp) {
        const long long units = (long long)rows * d.norm_parts;
        smc_launch_dep(ctx->use_pdl, kernel, dim3((unsigned)(warp ? (units + 7) / 8 : units)), dim3(256), 0, s, (const float *)b.y, g, b.ld, b.mix_norm,
                       static_cast<T *>(b.o), b.ldo, rows, inner, d.norm_parts, d.gate == SMC_GATE_SIGMOID, d.out_scale, d.eps);
    };
    const size_t at = 4 * sizeof(T) - 1;
    const bool four = n % 4 == 0 && b.ld % 4 == 0 && b.ldo % 4 == 0 && ((reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(b.o)) & at) == 0;
    if (n <= 512) four ? go(norm_gate_kernel<T, 4, true>, true) : go(norm_gate_kernel<T, 1, true>, true);
    else four ? go(norm_gate_kernel<T, 4, false>, false) : go(norm_gate_kernel<T, 1, false>, false);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

template <typename T>
int steps(smc_ctx *ctx, const smc_linear_dims &d, const smc_linear_bufs &b, const smc_rows &rw, cudaStream_t s)
{
    const bool seq = rw.seq0 >= 0;
    const int cap = seq ? (rw.n < SC ? rw.n : SC) : 1;
    const size_t smem = (size_t)cap * (2 * d.dim + 16) * sizeof(float);
    auto go = [&](auto kernel) {
        if (smem > 40 * 1024) SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(d.heads, (d.vdim + 15) / 16, seq ? 1 : rw.n), dim3(128), smem, s, static_cast<const T *>(b.in), b.ld, b.col,
                       b.y, b.state, rw, b.decay, b.cosT, b.sinT, b.max_seq, d.heads, d.vdim, d.dim, d.rot_dims, d.k_scale);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    if (d.dim % 4 == 0) {
        if (d.dim <= 32) return go(linear_step_kernel<T, 4, true>);
        if (d.dim <= 64) return go(linear_step_kernel<T, 8, true>);
        if (d.dim <= 128) return go(linear_step_kernel<T, 16, true>);
        if (d.dim <= 256) return go(linear_step_kernel<T, 32, true>);
        return go(linear_step_kernel<T, 64, true>);
    }
    if (d.dim <= 64) return go(linear_step_kernel<T, 8, false>);
    return go(linear_step_kernel<T, 64, false>);
}

// `finished`: the norm and gate are done as well
int chunks(smc_ctx *ctx, const smc_linear_dims &d, const smc_linear_bufs &b, const smc_rows &rw, bool &finished, cudaStream_t s)
{
    const bf16 *in = static_cast<const bf16 *>(b.in) + b.col;
    const int H = d.heads, N = d.dim, P = d.vdim, nch = (rw.n + CH - 1) / CH;
    const bf16 *q = in, *k = in + H * N, *v = in + 2 * H * N;
    size_t ldq = b.ld;
    if (d.rot_dims > 0) {
        const int half = d.rot_dims / 2;
        auto rotate = [&](auto kernel, int v) {
            smc_launch_dep(ctx->use_pdl, kernel, dim3((2 * H * ((N - half) / v) + 255) / 256, rw.n), dim3(256), 0, s, static_cast<const bf16 *>(b.in), b.ld, b.col,
                           static_cast<bf16 *>(b.qk), rw, b.cosT, b.sinT, b.max_seq, H, N, d.rot_dims);
        };
        half % 4 == 0 ? rotate(linear_rotate_kernel<4>, 4) : rotate(linear_rotate_kernel<1>, 1);  // (dim and the columns are whole eights here)
        SMC_LAUNCH_CHECK(ctx);
        q = static_cast<const bf16 *>(b.qk), k = q + H * N, ldq = 2 * (size_t)H * N;
    }
    const int ss = CH * row_ld(N) + 2 * CH * (PB + 8) * 2;
    auto state = [&](auto kernel) {
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, ss));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(nch, H, (P + PB - 1) / PB), dim3(CTH), ss, s, k, ldq, v, (size_t)b.ld, b.part, rw.n, b.log2_decay, H, P, N,
                       d.k_scale);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    int rc = N <= 64 ? state(linear_state_kernel<4>) : (N <= 128 ? state(linear_state_kernel<8>) : state(linear_state_kernel<16>));
    if (rc) return rc;
    const int pn4 = P * N / 4;
    smc_launch_dep(ctx->use_pdl, linear_carry_kernel, dim3((H * pn4 + 255) / 256), dim3(256), 0, s, reinterpret_cast<const float4 *>(b.part),
                   static_cast<uint2 *>(b.start), reinterpret_cast<float4 *>(b.state), rw, b.log2_decay, H, pn4);
    SMC_LAUNCH_CHECK(ctx);
    finished = d.norm_parts == H && P <= 128 && b.ldo % 2 == 0 && (reinterpret_cast<uintptr_t>(b.o) & 3) == 0;
    const OutArgs A{q, k, v, v + H * P, ldq, ldq, (size_t)b.ld, (size_t)b.ld, static_cast<const bf16 *>(b.start), b.y, static_cast<bf16 *>(b.o), b.ldo,
                    finished, d.gate == SMC_GATE_SIGMOID, b.mix_norm, d.k_scale, d.out_scale, d.eps};
    const int os = out_smem(P, N);
    auto out = [&](auto kernel) {
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, os));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(nch, H, (P + 127) / 128), dim3(CTH), os, s, A, rw, b.log2_decay, H, P, N);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    return P <= 64 ? out(linear_out_kernel<8>) : out(linear_out_kernel<16>);
}

template <typename T>
int mix(smc_ctx *ctx, const smc_linear_dims &d, const smc_linear_bufs &b, const smc_rows &rw, cudaStream_t s)
{
    if constexpr (std::is_same<T, bf16>::value) {
        const bool aligned = b.ld % 8 == 0 && b.col % 8 == 0 && (reinterpret_cast<uintptr_t>(b.in) & 15) == 0;
        if (rw.seq0 >= 0 && rw.n >= CHUNK_ROWS && b.part && aligned && smc_linear_chunks_supported(d)) {
            bool finished = false;
            int rc = chunks(ctx, d, b, rw, finished, s);
            return rc || finished ? rc : norm_gate<T>(ctx, d, b, rw.n, s);
        }
    }
    int rc = steps<T>(ctx, d, b, rw, s);
    return rc ? rc : norm_gate<T>(ctx, d, b, rw.n, s);
}

}  // namespace

bool smc_linear_chunks_supported(const smc_linear_dims &d) { return d.dim % 8 == 0 && d.vdim % 8 == 0 && d.dim <= 256 && out_smem(d.vdim, d.dim) <= 220 * 1024; }

int smc_linear_check(smc_ctx *ctx, const smc_linear_dims &d)
{
    if (d.dim > 512) return smc_fail(ctx, SMC_E_UNSUPPORTED, "linear attention: dim %d (up to 512 are built)", d.dim);
    if (d.rot_dims % 2 || d.rot_dims > d.dim) return smc_fail(ctx, SMC_E_UNSUPPORTED, "linear attention: %d rotated elements of %d", d.rot_dims, d.dim);
    return SMC_OK;
}

int smc_linear_mix(smc_ctx *ctx, const smc_linear_dims &d, const smc_linear_bufs &b, const smc_rows &rw, int is_bf16, cudaStream_t s)
{
    return is_bf16 ? mix<bf16>(ctx, d, b, rw, s) : mix<float>(ctx, d, b, rw, s);
}
