// Latent attention: queries, keys and values pass through low-rank latents, and the cache holds one compressed row per
// token (kv_rank elements, shared by all heads) plus one rotated key part.  Scores are (q_u . W_uk c + q_r . k_r) * scale
// over a sliding window, softmax with an optional per-head sink in the denominator, values W_uv c.
//
// Two forms of the same sums:
//   absorbed   q_u is carried through W_uk once per query (latent_absorb_kernel); scores and the weighted sum then run on
//              the compressed rows themselves, and W_uv is applied to the sum (latent_value_kernel).  One row is read per
//              key and no key or value is ever rebuilt: decoding, short portions, and everything in fp32.
//   expanded   the portion's visible keys and values are rebuilt per head by one matmul and attended on the tensor cores
//              (latent_prefill_kernel): a third of the arithmetic at prompt sizes.
// The cache is a ring: position p lives in row p % ring, ring >= window - 1 + the longest portion, so the rows a portion
// writes never displace one that its first query still sees.
#include <math.h>

#include <type_traits>
#include <vector>

#include "smc_mma.cuh"

namespace {

// ------------------------------------------------------------------------------ after the down projections
// A warp per (row, part): the query latent normed, or the key/value latent normed and the shared key part rotated, both
// straight into the cache.
template <typename T>
__global__ void __launch_bounds__(256) latent_post_kernel(const T *__restrict__ down, T *__restrict__ cq, T *__restrict__ cache, smc_rows rw,
                                                          const float *__restrict__ q_norm, const float *__restrict__ kv_norm,
                                                          const float *__restrict__ cosT, const float *__restrict__ sinT, int qr, int rk, int rd,
                                                          int ring, int max_seq, float eps)
{
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, wid = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int r = wid >> 1;
    if (r >= rw.n) return;
    const T *src = down + (size_t)r * (qr + rk + rd);
    const bool kv = wid & 1;
    const int n = kv ? rk : qr;
    if (kv) src += qr;
    float ss = 0.f;
    for (int i = lane; i < n; i += 32) {
        const float v = to_f(src[i]);
        ss = fmaf(v, v, ss);
    }
    ss = smc_group_sum<32>(ss);
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)n) + eps));
    int slot, p;
    row_place(rw, r, slot, p);
    T *dst = kv ? cache + ((size_t)slot * ring + p % ring) * (rk + rd) : cq + (size_t)r * qr;
    const float *w = kv ? kv_norm : q_norm;
    for (int i = lane; i < n; i += 32) dst[i] = from_f<T>((to_f(src[i]) * inv) * w[i]);
    if (!kv) return;
    const int half = rd / 2;
    const size_t t = (size_t)min(p, max_seq - 1) * half;
    for (int i = lane; i < half; i += 32) {
        const float u = to_f(src[rk + i]), v = to_f(src[rk + half + i]), c = cosT[t + i], s = sinT[t + i];
        dst[rk + i] = from_f<T>(__fsub_rn(__fmul_rn(u, c), __fmul_rn(v, s)));
        dst[rk + half + i] = from_f<T>(__fadd_rn(__fmul_rn(v, c), __fmul_rn(u, s)));
    }
}

// ------------------------------------------------------------------------------ absorbed form
// qa[row, h] = [ W_uk[h]^T q_u | rotated q_r ], fp32.  CTA: one head, 64 latent columns, up to 8 rows; the warps split the
// sum over the head's unrotated elements.
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const T *__restrict__ q, const bf16 *__restrict__ wuk, float *__restrict__ qa, smc_rows rw,
                                                            const float *__restrict__ cosT, const float *__restrict__ sinT, int heads, int dim, int rd,
                                                            int rk, int max_seq)
{
    extern __shared__ float sq[];  // [8][dim]
    __shared__ float red[8][8][64];
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.x, r0 = blockIdx.z * 8, nr = min(8, rw.n - r0);
    const int hw = dim + rd;
    for (int e = threadIdx.x; e < nr * dim; e += 256) sq[e] = to_f(q[((size_t)(r0 + e / dim) * heads + h) * hw + e % dim]);
    for (int e = nr * dim + threadIdx.x; e < 8 * dim; e += 256) sq[e] = 0.f;
    __syncthreads();
    const int ca = blockIdx.y * 64 + lane, cb = ca + 32;
    float acc[8][2];
#pragma unroll
    for (int m = 0; m < 8; ++m) acc[m][0] = acc[m][1] = 0.f;
    const bf16 *wp = wuk + (size_t)h * dim * rk;
#pragma unroll 4
    for (int d = warp; d < dim; d += 8) {
        const float wa = ca < rk ? to_f(wp[(size_t)d * rk + ca]) : 0.f, wb = cb < rk ? to_f(wp[(size_t)d * rk + cb]) : 0.f;
#pragma unroll
        for (int m = 0; m < 8; ++m) {
            const float v = sq[m * dim + d];
            acc[m][0] = fmaf(v, wa, acc[m][0]), acc[m][1] = fmaf(v, wb, acc[m][1]);
        }
    }
#pragma unroll
    for (int m = 0; m < 8; ++m) red[warp][m][lane] = acc[m][0], red[warp][m][lane + 32] = acc[m][1];
    __syncthreads();
    for (int e = threadIdx.x; e < nr * 64; e += 256) {
        const int m = e >> 6, c = e & 63;
        if (blockIdx.y * 64 + c >= rk) continue;
        float v = red[0][m][c];
#pragma unroll
        for (int i = 1; i < 8; ++i) v += red[i][m][c];
        qa[((size_t)(r0 + m) * heads + h) * (rk + rd) + blockIdx.y * 64 + c] = v;
    }
    if (blockIdx.y) return;
    const int half = rd / 2;
    for (int e = threadIdx.x; e < nr * half; e += 256) {
        const int m = e / half, i = e % half;
        int slot, p;
        row_place(rw, r0 + m, slot, p);
        const T *src = q + ((size_t)(r0 + m) * heads + h) * hw + dim;
        const size_t t = (size_t)min(p, max_seq - 1) * half + i;
        const float u = to_f(src[i]), v = to_f(src[half + i]), c = cosT[t], s = sinT[t];
        float *dst = qa + ((size_t)(r0 + m) * heads + h) * (rk + rd) + rk;
        dst[i] = __fsub_rn(__fmul_rn(u, c), __fmul_rn(v, s));
        dst[half + i] = __fadd_rn(__fmul_rn(v, c), __fmul_rn(u, s));
    }
}

// oc[row, h] = sum over the window of softmax weight * compressed row; one CTA per (head, row), the warps take every
// eighth key with a running maximum each and are merged at the end, together with the sink.
template <typename T, int EPL>
__global__ void __launch_bounds__(256) latent_attend_kernel(const float *__restrict__ qa, const T *__restrict__ cache, float *__restrict__ oc,
                                                            smc_rows rw, const float *__restrict__ sink, int heads, int rk, int rd, int ring,
                                                            int window, float scale)
{
    extern __shared__ float sm[];  // query [rk + rd], then partial sums [8][rk]
    __shared__ float sm_m[8], sm_l[8];
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.x, r = blockIdx.y, row = rk + rd;
    float *qs = sm, *part = sm + row;
    for (int i = threadIdx.x; i < row; i += 256) qs[i] = qa[((size_t)r * heads + h) * row + i];
    __syncthreads();
    int slot, p;
    row_place(rw, r, slot, p);
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    const T *base = cache + (size_t)slot * ring * row;
    float o[EPL], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int j = 0; j < EPL; ++j) o[j] = 0.f;
    for (int k = lo + warp; k <= p; k += 8) {
        const T *kr = base + (size_t)(k % ring) * row;
        float c[EPL], s = 0.f;
#pragma unroll
        for (int j = 0; j < EPL; ++j) {
            const int i = lane + 32 * j;
            c[j] = i < rk ? to_f(kr[i]) : 0.f;
            if (i < rk) s = fmaf(qs[i], c[j], s);
        }
        for (int i = rk + lane; i < row; i += 32) s = fmaf(qs[i], to_f(kr[i]), s);
        s = smc_group_sum<32>(s) * scale;
        const float nm = fmaxf(m, s), f = expf(m - nm), e = expf(s - nm);
        l = fmaf(l, f, e), m = nm;
#pragma unroll
        for (int j = 0; j < EPL; ++j) o[j] = fmaf(e, c[j], o[j] * f);
    }
#pragma unroll
    for (int j = 0; j < EPL; ++j)
        if (lane + 32 * j < rk) part[warp * rk + lane + 32 * j] = o[j];
    if (lane == 0) sm_m[warp] = m, sm_l[warp] = l;
    __syncthreads();
    float top = sink ? sink[h] : -INFINITY;
#pragma unroll
    for (int w = 0; w < 8; ++w) top = fmaxf(top, sm_m[w]);
    float f[8], den = sink ? expf(sink[h] - top) : 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) f[w] = expf(sm_m[w] - top), den = fmaf(f[w], sm_l[w], den);
    const float inv = __fdiv_rn(1.0f, den);
    for (int i = threadIdx.x; i < rk; i += 256) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v = fmaf(f[w], part[w * rk + i], v);
        oc[((size_t)r * heads + h) * rk + i] = v * inv;
    }
}

// o[row, h, v] = W_uv[h, v] . oc[row, h]: a warp per output element, up to 8 rows.
template <typename T>
__global__ void __launch_bounds__(256) latent_value_kernel(const float *__restrict__ oc, const bf16 *__restrict__ wuv, T *__restrict__ o, int rows,
                                                           int heads, int vdim, int rk)
{
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, n = blockIdx.x * 8 + (threadIdx.x >> 5), r0 = blockIdx.y * 8, nr = min(8, rows - r0);
    if (n >= heads * vdim) return;
    const int h = n / vdim;
    const bf16 *w = wuv + (size_t)n * rk;
    float acc[8];
#pragma unroll
    for (int m = 0; m < 8; ++m) acc[m] = 0.f;
    for (int i = lane; i < rk; i += 32) {
        const float wv = to_f(w[i]);
#pragma unroll
        for (int m = 0; m < 8; ++m)
            if (m < nr) acc[m] = fmaf(wv, oc[((size_t)(r0 + m) * heads + h) * rk + i], acc[m]);
    }
#pragma unroll
    for (int m = 0; m < 8; ++m) {
        const float v = smc_group_sum<32>(acc[m]);
        if (lane == 0 && m < nr) o[(size_t)(r0 + m) * heads * vdim + n] = from_f<T>(v);
    }
}

// ------------------------------------------------------------------------------ expanded form (bfloat16)
// The rows a portion can see, oldest first: keys[j] = cache row of position k0 + j.
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4 *__restrict__ cache, uint4 *__restrict__ keys, int slot, int k0, int n, int ring,
                                                            int row16)
{
    smc_grid_dep_sync();
    const long long e = (long long)blockIdx.x * 256 + threadIdx.x;
    if (e >= (long long)n * row16) return;
    const int j = (int)(e / row16), c = (int)(e % row16);
    keys[e] = cache[((size_t)slot * ring + (k0 + j) % ring) * row16 + c];
}

// ------------------------------------------------------------------------------ absorbed form on the tensor cores (bfloat16)
// One row, up to 16 heads per cluster of up to eight CTAs; each CTA takes every cluster-size-th 64-key tile of the window and
// the cluster merges its partial sums through distributed shared memory.  The absorbed query (fp32) enters as a bfloat16 pair hi + lo,
// so scores keep 16 bits of it; the cached rows are exact operands of both products.  All heads read the same keys: a tile
// is fetched once per 16 heads.
// Scores split their sum over the latent across eight warps (twice, for the halves of a tile): a warp keeps its slice of the query in registers for all tiles and
// reads its slice of every key once; the eight partial score tiles meet in shared memory.
//   shared memory: query planes [2][16][ldk], later the partial scores [8][16][72] fp32; two key tiles [64][ldk]; weights
//   [16][72] bfloat16
// The keys and the position are fetched BEFORE the wait for the predecessor: they were written by the kernel before it, and a
// kernel that is launched early is so only after every CTA of its predecessor has passed its own wait.
constexpr int DT = 64, DCL = 8, KPW = 5, DTH = 512, DLS = 72;  // keys per tile, largest cluster, 16-element slices of the sum per warp, threads, score row
__host__ __device__ inline int decode_head_bytes(int ldk) { return 2 * 16 * ldk > 8 * 16 * DLS * 4 ? 2 * 16 * ldk : 8 * 16 * DLS * 4; }
template <int OPW>  // 16-column groups of the latent a warp accumulates (16 warps)
__global__ void __launch_bounds__(DTH)
latent_decode_kernel(const float *__restrict__ qa, const bf16 *__restrict__ q, const bf16 *__restrict__ cache, bf16 *__restrict__ oc, smc_rows rw,
                     const float *__restrict__ sink, const float *__restrict__ cosT, const float *__restrict__ sinT, int heads, int dim, int rk, int rd,
                     int ring, int window, float scale, int max_seq)
{
    extern __shared__ __align__(16) uint8_t sm_raw[];
    __shared__ float row_m[16], row_l[16], row_f[16], all_m[DCL][16], all_l[DCL][16], all_f[DCL][16];
    const int row = rk + rd, row16 = (row + 15) & ~15, ldk = (row16 + 8) * 2;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int rank = blockIdx.x, h0 = blockIdx.y * 16, nh = min(16, heads - h0), r = blockIdx.z;
    uint8_t *q_s = sm_raw, *k_s = q_s + decode_head_bytes(ldk), *p_s = k_s + 2 * DT * ldk;
    const uint32_t qb = (uint32_t)__cvta_generic_to_shared(q_s), kb = (uint32_t)__cvta_generic_to_shared(k_s), pb = (uint32_t)__cvta_generic_to_shared(p_s);
    float *sc = reinterpret_cast<float *>(q_s);
    const int cl = gridDim.x;
    // padding columns of the planes and tiles, and the planes' rows without a head
    const int pad = ldk / 2 - row;
    for (int e = threadIdx.x; e < (2 * 16 + 2 * DT) * pad; e += DTH) {
        const int j = e / pad;
        reinterpret_cast<bf16 *>(j < 32 ? q_s + j * ldk : k_s + (j - 32) * ldk)[row + e % pad] = __float2bfloat16_rn(0.f);
    }
    for (int e = threadIdx.x; e < 2 * (16 - nh) * row; e += DTH) {
        const int rr = e / row, pl = rr / (16 - nh);
        reinterpret_cast<bf16 *>(sm_raw + (pl * 16 + nh + rr % (16 - nh)) * ldk)[e % row] = __float2bfloat16_rn(0.f);
    }
    int slot, p;
    row_place(rw, r, slot, p);
    const int lo = window > 0 ? max(0, p - window + 1) : 0, n = p - lo + 1, tiles = (n + DT - 1) / DT;
    const bf16 *base = cache + (size_t)slot * ring * row;
    const int chunks = row / 8, lo_row = lo % ring;
    auto fetch = [&](int t, int buf) {  // a warp per row
        for (int j = warp; j < DT; j += DTH / 32) {
            const int k = t * DT + j;
            const bool in = k < n;
            int rr = lo_row + (in ? k : 0);
            rr -= rr >= ring ? ring : 0;  // n <= ring
            const bf16 *src = base + (size_t)rr * row;
            for (int c = lane; c < chunks; c += 32) cp16(kb + (uint32_t)((buf * DT + j) * ldk + 16 * c), src + 8 * c, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (rank < tiles) fetch(rank, 0);
    smc_grid_dep_sync();
    auto put_q = [&](int hh, int i, float v) {
        const bf16 hi = __float2bfloat16_rn(v);
        reinterpret_cast<bf16 *>(q_s + hh * ldk)[i] = hi;
        reinterpret_cast<bf16 *>(q_s + (16 + hh) * ldk)[i] = __float2bfloat16_rn(v - __bfloat162float(hi));
    };
    for (int hh = warp; hh < nh; hh += DTH / 32) {
        const float4 *src = reinterpret_cast<const float4 *>(qa + ((size_t)r * heads + h0 + hh) * rk);
#pragma unroll 4
        for (int i = lane; i < rk / 4; i += 32) {
            const float4 v = src[i];
            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
            const __nv_bfloat162 c = __floats2bfloat162_rn(v.x - __bfloat162float(a.x), v.y - __bfloat162float(a.y)),
                                 d = __floats2bfloat162_rn(v.z - __bfloat162float(b.x), v.w - __bfloat162float(b.y));
            *reinterpret_cast<uint2 *>(q_s + hh * ldk + 8 * i) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
            *reinterpret_cast<uint2 *>(q_s + (16 + hh) * ldk + 8 * i) = make_uint2(*reinterpret_cast<const uint32_t *>(&c), *reinterpret_cast<const uint32_t *>(&d));
        }
    }
    const int half = rd / 2;
    for (int e = threadIdx.x; e < nh * half; e += DTH) {
        const int hh = e / half, i = e % half;
        const bf16 *src = q + ((size_t)r * heads + h0 + hh) * (dim + rd) + dim;
        const size_t ti = (size_t)min(p, max_seq - 1) * half + i;
        const float u = to_f(src[i]), v = to_f(src[half + i]), c = cosT[ti], s = sinT[ti];
        put_q(hh, rk + i, __fsub_rn(__fmul_rn(u, c), __fmul_rn(v, s)));
        put_q(hh, rk + half + i, __fadd_rn(__fmul_rn(v, c), __fmul_rn(u, s)));
    }
    if (threadIdx.x < 16) row_m[threadIdx.x] = -INFINITY, row_l[threadIdx.x] = 0.f;
    float o[2 * OPW][4];
#pragma unroll
    for (int i = 0; i < 2 * OPW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    __syncthreads();
    // this warp's slice of the query
    uint32_t ah[KPW][4], al[KPW][4];
    const int ksteps = row16 / 16, kpw = (ksteps + 7) / 8, ks0 = (warp & 7) * kpw, khalf = (warp >> 3) * (DT / 2), nks = max(0, min(kpw, ksteps - ks0));
#pragma unroll
    for (int i = 0; i < KPW; ++i) {
        ah[i][0] = ah[i][1] = ah[i][2] = ah[i][3] = al[i][0] = al[i][1] = al[i][2] = al[i][3] = 0u;
        if (i < nks) {
            const uint32_t a = qb + (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + 16 * (lane >> 4) + 32 * (ks0 + i));
            ldsm4(a, ah[i]);
            ldsm4(a + 16 * ldk, al[i]);
        }
    }
    __syncthreads();  // the planes make room for the partial scores
    int buf = 0;
    for (int t = rank; t < tiles; t += cl, buf ^= 1) {
        if (t + cl < tiles) {
            fetch(t + cl, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        // ---- partial scores of half of the keys
        {
            float s[DT / 16][4];
#pragma unroll
            for (int i = 0; i < DT / 16; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
            const uint32_t bk = kb + (uint32_t)((buf * DT + khalf + (lane & 7) + 8 * (lane >> 4)) * ldk + 16 * ((lane >> 3) & 1) + 32 * ks0);
#pragma unroll
            for (int i = 0; i < KPW; ++i)
                if (i < nks) {
#pragma unroll
                    for (int np = 0; np < DT / 32; ++np) {
                        uint32_t b[4];
                        ldsm4(bk + (uint32_t)(np * 16 * ldk + 32 * i), b);
                        mma_bf16(s[2 * np], al[i], b[0], b[1]), mma_bf16(s[2 * np + 1], al[i], b[2], b[3]);
                        mma_bf16(s[2 * np], ah[i], b[0], b[1]), mma_bf16(s[2 * np + 1], ah[i], b[2], b[3]);
                    }
                }
            float *d = sc + ((warp & 7) * 16 + g) * DLS + khalf + 2 * tg;
#pragma unroll
            for (int i = 0; i < DT / 16; ++i) {
                *reinterpret_cast<float2 *>(d + 8 * i) = make_float2(s[i][0], s[i][1]);
                *reinterpret_cast<float2 *>(d + 8 * DLS + 8 * i) = make_float2(s[i][2], s[i][3]);
            }
        }
        __syncthreads();
        // ---- running softmax: a head per warp
        {
            float s0 = 0.f, s1 = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) s0 += sc[(w * 16 + warp) * DLS + lane], s1 += sc[(w * 16 + warp) * DLS + lane + 32];
            s0 = t * DT + lane < n ? s0 * scale : -INFINITY, s1 = t * DT + lane + 32 < n ? s1 * scale : -INFINITY;
            const float before = row_m[warp];
            float m = fmaxf(s0, s1);
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
            m = fmaxf(m, before);  // every tile holds a key, so the maximum is finite
            const float e0 = expf(s0 - m), e1 = expf(s1 - m);
            const float l = smc_group_sum<32>(e0 + e1);
            bf16 *pp = reinterpret_cast<bf16 *>(p_s) + warp * 72;
            pp[lane] = __float2bfloat16_rn(e0), pp[lane + 32] = __float2bfloat16_rn(e1);
            if (lane == 0) {
                const float f = expf(before - m);
                row_f[warp] = f, row_m[warp] = m, row_l[warp] = fmaf(row_l[warp], f, l);
            }
        }
        __syncthreads();
        const float f0 = row_f[g], f1 = row_f[g + 8];
#pragma unroll
        for (int i = 0; i < 2 * OPW; ++i) o[i][0] *= f0, o[i][1] *= f0, o[i][2] *= f1, o[i][3] *= f1;
#pragma unroll
        for (int ks = 0; ks < DT / 16; ++ks) {
            uint32_t a[4];
            ldsm4(pb + (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * 144 + 16 * (lane >> 4) + 32 * ks), a);
#pragma unroll
            for (int i = 0; i < OPW; ++i) {
                const int grp = warp + DTH / 32 * i;
                if (16 * grp < rk) {
                    uint32_t b[4];
                    ldsm4t(kb + (uint32_t)((buf * DT + ks * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + 32 * grp + 16 * (lane >> 4)), b);
                    mma_bf16(o[2 * i], a, b[0], b[1]);
                    mma_bf16(o[2 * i + 1], a, b[2], b[3]);
                }
            }
        }
        __syncthreads();  // the tile buffer, scores and weights are rewritten next
    }
    // ---- merge over the cluster: partial sums [16][rk] fp32 over the key tiles' space
    float *part = reinterpret_cast<float *>(k_s);
    const int ldp = rk + 4;
#pragma unroll
    for (int i = 0; i < OPW; ++i) {
        const int grp = warp + DTH / 32 * i;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int c = 16 * grp + 8 * j + 2 * tg;
            if (c < rk) {
                part[g * ldp + c] = o[2 * i + j][0], part[(g + 8) * ldp + c] = o[2 * i + j][2];
                if (c + 1 < rk) part[g * ldp + c + 1] = o[2 * i + j][1], part[(g + 8) * ldp + c + 1] = o[2 * i + j][3];
            }
        }
    }
    auto cluster_sync = [] { asm volatile("barrier.cluster.arrive;\n\tbarrier.cluster.wait;" ::: "memory"); };
    cluster_sync();
    auto remote = [](const void *ptr, int cta) {
        uint32_t a = (uint32_t)__cvta_generic_to_shared(ptr), v;
        float f;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(v) : "r"(a), "r"(cta));
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(f) : "r"(v) : "memory");
        return f;
    };
    if (threadIdx.x < DCL * 16) {
        const int k = threadIdx.x >> 4, hh = threadIdx.x & 15;
        all_m[k][hh] = k < cl ? remote(&row_m[hh], k) : -INFINITY, all_l[k][hh] = k < cl ? remote(&row_l[hh], k) : 0.f;
    }
    __syncthreads();
    if (threadIdx.x < 16) {
        const int hh = threadIdx.x;
        const float sk = sink && hh < nh ? sink[h0 + hh] : -INFINITY;
        float top = sk;
#pragma unroll
        for (int k = 0; k < DCL; ++k) top = fmaxf(top, all_m[k][hh]);
        float den = sink ? expf(sk - top) : 0.f;
#pragma unroll
        for (int k = 0; k < DCL; ++k) all_f[k][hh] = expf(all_m[k][hh] - top), den = fmaf(all_f[k][hh], all_l[k][hh], den);
#pragma unroll
        for (int k = 0; k < DCL; ++k) all_f[k][hh] = __fdiv_rn(all_f[k][hh], den);
    }
    __syncthreads();
    const int per = (rk + cl - 1) / cl, c0 = rank * per, c1 = min(rk, c0 + per);
    for (int e = threadIdx.x; e < nh * per; e += DTH) {
        const int hh = e / per, c = c0 + e % per;
        if (c >= c1) continue;
        float x[DCL], v = 0.f;
#pragma unroll
        for (int k = 0; k < DCL; ++k) x[k] = k < cl ? remote(&part[hh * ldp + c], k) : 0.f;  // zeros from a CTA without a tile, its factor is zero too
#pragma unroll
        for (int k = 0; k < DCL; ++k) v = fmaf(all_f[k][hh], x[k], v);
        oc[((size_t)r * heads + h0 + hh) * rk + c] = __float2bfloat16_rn(v);
    }
    cluster_sync();  // nobody leaves while its sums are read
}

size_t decode_smem(const smc_latent_dims &d)
{
    const int row16 = (d.kv_rank + d.rot_dim + 15) & ~15, ldk = (row16 + 8) * 2;
    const size_t tiles = (size_t)2 * DT * ldk, merged = (size_t)16 * (d.kv_rank + 4) * 4;
    return decode_head_bytes(ldk) + (tiles > merged ? tiles : merged) + 16 * 72 * 2 + 64;
}

// ukt[h][c][d] = W_uk[h * dim + d][c]
__global__ void __launch_bounds__(256) transpose_uk_kernel(const bf16 *__restrict__ wuk, bf16 *__restrict__ ukt, int heads, int dim, int rk)
{
    const size_t e = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (e >= (size_t)heads * dim * rk) return;
    const int d = (int)(e % dim), c = (int)(e / dim % rk), h = (int)(e / ((size_t)dim * rk));
    ukt[e] = wuk[((size_t)h * dim + d) * rk + c];
}

// 64 query rows of one head per CTA (16 per warp), key tiles of 64, two tile buffers filled by cp.async.  Scores and the
// running softmax are fp32; the weights enter the second product as bfloat16.  Head sizes are padded to 16 with zeros in
// shared memory.  VT: value tiles of 8 columns a thread keeps accumulators for.
template <int VT>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const bf16 *__restrict__ q, const bf16 *__restrict__ keys, const bf16 *__restrict__ kv,
                                                             bf16 *__restrict__ out, const float *__restrict__ sink, const float *__restrict__ cosT,
                                                             const float *__restrict__ sinT, int T, int nk, int pos0, int k0, int heads, int dim,
                                                             int rd, int vdim, int rk, int window, float scale, int max_seq)
{
    constexpr int QR = 64, KT = 64;
    const int qk = dim + rd, qk16 = (qk + 15) & ~15, v16 = (vdim + 15) & ~15;
    const int ldk = (qk16 + 8) * 2, ldv = (v16 + 8) * 2;  // bytes per row: an odd number of 16-byte units
    extern __shared__ __align__(16) uint8_t sm_raw[];
    const uint32_t sq = (uint32_t)__cvta_generic_to_shared(sm_raw), sk = sq + QR * ldk, sv = sk + 2 * KT * ldk;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int h = blockIdx.x, t0 = (int)(gridDim.y - 1 - blockIdx.y) * QR;
    // padding columns are never written by the copies below: clear everything once
    for (uint32_t e = threadIdx.x; e < (uint32_t)(QR * ldk + 2 * KT * (ldk + ldv)) / 16; e += 128)
        reinterpret_cast<uint4 *>(sm_raw)[e] = make_uint4(0u, 0u, 0u, 0u);
    smc_grid_dep_sync();
    __syncthreads();

    const int p_first = pos0 + t0, p_last = pos0 + min(T, t0 + QR) - 1;            // positions of the CTA's queries
    const int key_lo = (window > 0 ? max(0, p_first - window + 1) : 0) - k0;        // keys as indices from k0
    const int key_hi = p_last - k0;                                                // inclusive; < nk
    const int ldkv = heads * (dim + vdim), ldc = rk + rd;
    const int cu = dim / 8, cr = rd / 8, cv = vdim / 8;
    // rows of a matrix piece -> tile, 16 bytes per thread and copy; keys past the last visible one become zeros
    auto copy = [&](uint32_t dst, int ldd, const bf16 *src, int lds, int pieces, int lanes, int start) {
        const int c0 = threadIdx.x & (lanes - 1), j0 = threadIdx.x / lanes, js = 128 / lanes;
        for (int c = c0; c < pieces; c += lanes) {
            const bf16 *p = src + (size_t)(start + j0) * lds + 8 * c;
            uint32_t d = dst + (uint32_t)(j0 * ldd + 16 * c);
#pragma unroll 4
            for (int j = j0; j < KT; j += js, p += (size_t)js * lds, d += (uint32_t)(js * ldd)) {
                const bool in = start + j <= key_hi;
                cp16(d, in ? p : src, in);
            }
        }
    };
    auto fetch = [&](int start, int buf) {
        const uint32_t kb = sk + (uint32_t)buf * KT * ldk, vb = sv + (uint32_t)buf * KT * ldv;
        copy(kb, ldk, kv + h * dim, ldkv, cu, 16, start);
        copy(kb + 16 * cu, ldk, keys + rk, ldc, cr, 8, start);
        copy(vb, ldv, kv + heads * dim + h * vdim, ldkv, cv, 16, start);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(key_lo, 0);
    // ---- the query tile, its last rd elements rotated
    for (int e = threadIdx.x; e < QR * cu; e += 128) {
        const int r = e / cu, c = e % cu;
        if (t0 + r < T)
            *reinterpret_cast<uint4 *>(sm_raw + r * ldk + 16 * c) = *reinterpret_cast<const uint4 *>(q + ((size_t)(t0 + r) * heads + h) * qk + 8 * c);
    }
    const int half = rd / 2;
    for (int e = threadIdx.x; e < QR * half; e += 128) {
        const int r = e / half, i = e % half;
        if (t0 + r >= T) continue;
        const bf16 *src = q + ((size_t)(t0 + r) * heads + h) * qk + dim;
        const size_t ti = (size_t)min(p_first + r, max_seq - 1) * half + i;
        const float u = to_f(src[i]), v = to_f(src[half + i]), c = cosT[ti], s = sinT[ti];
        bf16 *dst = reinterpret_cast<bf16 *>(sm_raw + r * ldk) + dim;
        dst[i] = __float2bfloat16_rn(__fsub_rn(__fmul_rn(u, c), __fmul_rn(v, s)));
        dst[half + i] = __float2bfloat16_rn(__fadd_rn(__fmul_rn(v, c), __fmul_rn(u, s)));
    }

    const int tile_hi = p_first - k0, tile_lo = window > 0 ? p_first + QR - window - k0 : -k0;  // keys all of the CTA's queries see
    // rows g and g + 8 of the warp's sixteen; the keys each sees, as indices
    const int r0 = warp * 16 + g, r1 = r0 + 8;
    int hi0 = -1, hi1 = -1, lo0 = 0, lo1 = 0;
    if (t0 + r0 < T) hi0 = p_first + r0 - k0, lo0 = window > 0 ? max(0, p_first + r0 - window + 1) - k0 : -k0;
    if (t0 + r1 < T) hi1 = p_first + r1 - k0, lo1 = window > 0 ? max(0, p_first + r1 - window + 1) - k0 : -k0;
    constexpr float LOG2E = 1.4426950408889634f;
    const float scale2 = scale * LOG2E;  // scores, maxima and the sink in powers of two
    const float s0 = sink ? sink[h] * LOG2E : -INFINITY;
    float m0 = s0, m1 = s0, l0 = sink ? 1.f : 0.f, l1 = l0;
    // (with a sink the running pair (maximum, sum) starts as that of the one extra term)
    float o[VT][4];
#pragma unroll
    for (int n = 0; n < VT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const uint32_t a_off = sq + (uint32_t)((warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + 16 * (lane >> 4));
    const uint32_t bk_off = (uint32_t)(((lane & 7) + 8 * (lane >> 4)) * ldk + 16 * ((lane >> 3) & 1));
    const uint32_t bv_off = (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * ldv + 16 * (lane >> 4));

    int buf = 0;
    for (int start = key_lo; start <= key_hi; start += KT, buf ^= 1) {
        if (start + KT <= key_hi) {
            fetch(start + KT, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t kb = sk + (uint32_t)buf * KT * ldk + bk_off, vb = sv + (uint32_t)buf * KT * ldv + bv_off;
        float s[KT / 8][4];
#pragma unroll
        for (int n = 0; n < KT / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll 4
        for (int ks = 0; ks < qk16 / 16; ++ks) {
            uint32_t a[4];
            ldsm4(a_off + 32 * ks, a);
#pragma unroll
            for (int np = 0; np < KT / 16; ++np) {
                uint32_t b[4];
                ldsm4(kb + np * 16 * ldk + 32 * ks, b);
                mma_bf16(s[2 * np], a, b[0], b[1]);
                mma_bf16(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        float tm0 = -INFINITY, tm1 = -INFINITY;
        if (start >= tile_lo && start + KT - 1 <= tile_hi) {  // every query of the CTA sees the whole tile
#pragma unroll
            for (int n = 0; n < KT / 8; ++n) {
                s[n][0] *= scale2, s[n][1] *= scale2, s[n][2] *= scale2, s[n][3] *= scale2;
                tm0 = fmaxf(tm0, fmaxf(s[n][0], s[n][1])), tm1 = fmaxf(tm1, fmaxf(s[n][2], s[n][3]));
            }
        } else {
#pragma unroll
            for (int n = 0; n < KT / 8; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int key = start + 8 * n + 2 * tg + i;
                    s[n][i] = key >= lo0 && key <= hi0 ? s[n][i] * scale2 : -INFINITY;
                    s[n][2 + i] = key >= lo1 && key <= hi1 ? s[n][2 + i] * scale2 : -INFINITY;
                    tm0 = fmaxf(tm0, s[n][i]), tm1 = fmaxf(tm1, s[n][2 + i]);
                }
            }
        }
        tm0 = fmaxf(tm0, __shfl_xor_sync(0xffffffffu, tm0, 1)), tm0 = fmaxf(tm0, __shfl_xor_sync(0xffffffffu, tm0, 2));
        tm1 = fmaxf(tm1, __shfl_xor_sync(0xffffffffu, tm1, 1)), tm1 = fmaxf(tm1, __shfl_xor_sync(0xffffffffu, tm1, 2));
        const float nm0 = fmaxf(m0, tm0), nm1 = fmaxf(m1, tm1);
        // a row that has seen nothing yet keeps maximum -inf; its weights are 0
        const float b0 = nm0 > -INFINITY ? nm0 : 0.f, b1 = nm1 > -INFINITY ? nm1 : 0.f;
        const float c0 = ex2(m0 - b0), c1 = ex2(m1 - b1);
        float ps0 = 0.f, ps1 = 0.f;
        uint32_t p[KT / 16][4];
#pragma unroll
        for (int n = 0; n < KT / 8; ++n) {
            const float e0 = ex2(s[n][0] - b0), e1 = ex2(s[n][1] - b0), e2 = ex2(s[n][2] - b1), e3 = ex2(s[n][3] - b1);
            ps0 += e0 + e1, ps1 += e2 + e3;
            p[n >> 1][(n & 1) * 2] = pack2(e0, e1), p[n >> 1][(n & 1) * 2 + 1] = pack2(e2, e3);
        }
        ps0 += __shfl_xor_sync(0xffffffffu, ps0, 1), ps0 += __shfl_xor_sync(0xffffffffu, ps0, 2);
        ps1 += __shfl_xor_sync(0xffffffffu, ps1, 1), ps1 += __shfl_xor_sync(0xffffffffu, ps1, 2);
        l0 = fmaf(l0, c0, ps0), l1 = fmaf(l1, c1, ps1);
        m0 = nm0, m1 = nm1;
#pragma unroll
        for (int n = 0; n < VT; ++n) o[n][0] *= c0, o[n][1] *= c0, o[n][2] *= c1, o[n][3] *= c1;
#pragma unroll
        for (int j = 0; j < KT / 16; ++j)
#pragma unroll
            for (int np = 0; np < VT / 2; ++np)
                if (16 * np < v16) {
                    uint32_t b[4];
                    ldsm4t(vb + j * 16 * ldv + 32 * np, b);
                    mma_bf16(o[2 * np], p[j], b[0], b[1]);
                    mma_bf16(o[2 * np + 1], p[j], b[2], b[3]);
                }
        __syncthreads();  // the buffer is refilled by the next iteration's fetch
    }
    const float i0 = l0 > 0.f ? __fdiv_rn(1.0f, l0) : 0.f, i1 = l1 > 0.f ? __fdiv_rn(1.0f, l1) : 0.f;
#pragma unroll
    for (int n = 0; n < VT; ++n) {
        const int c = 8 * n + 2 * tg;
        if (c >= vdim) continue;
        if (t0 + r0 < T) *reinterpret_cast<uint32_t *>(out + ((size_t)(t0 + r0) * heads + h) * vdim + c) = pack2(o[n][0] * i0, o[n][1] * i0);
        if (t0 + r1 < T) *reinterpret_cast<uint32_t *>(out + ((size_t)(t0 + r1) * heads + h) * vdim + c) = pack2(o[n][2] * i1, o[n][3] * i1);
    }
}

size_t prefill_smem(const smc_latent_dims &d)
{
    const int ldk = (((d.dim + d.rot_dim + 15) & ~15) + 8) * 2, ldv = (((d.vdim + 15) & ~15) + 8) * 2;
    return (size_t)64 * ldk + 2 * 64 * (size_t)(ldk + ldv);
}

// portions from this many rows on take the expanded form
constexpr int EXPAND_ROWS = 17;

template <typename T>
int attend_rows(smc_ctx *ctx, const smc_latent_dims &d, const smc_latent_bufs &b, const smc_rows &rw, const float *sink, cudaStream_t s)
{
    const int row = d.kv_rank + d.rot_dim;
    const size_t smem = ((size_t)row + 8 * d.kv_rank) * sizeof(float);
#define SMC_ATTEND(E)                                                                                                                        \
    do {                                                                                                                                     \
        if (smem > 40 * 1024)                                                                                                                \
            SMC_CUDA(ctx, cudaFuncSetAttribute(latent_attend_kernel<T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));         \
        smc_launch_dep(ctx->use_pdl, latent_attend_kernel<T, E>, dim3(d.heads, rw.n), dim3(256), smem, s, (const float *)b.qa,               \
                       static_cast<const T *>(b.cache), static_cast<float *>(b.oc), rw, sink, d.heads, d.kv_rank, d.rot_dim, d.ring, d.window, d.scale);           \
    } while (0)
    if (d.kv_rank <= 64) SMC_ATTEND(2);
    else if (d.kv_rank <= 128) SMC_ATTEND(4);
    else if (d.kv_rank <= 256) SMC_ATTEND(8);
    else if (d.kv_rank <= 512) SMC_ATTEND(16);
    else SMC_ATTEND(32);
#undef SMC_ATTEND
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

// the same on the tensor cores: absorb, attend, rebuild the values
int attend_absorbed_mma(smc_ctx *ctx, const smc_latent_dims &d, const smc_latent_bufs &b, const smc_rows &rw, const smc_weight *w_ukv, const float *sink,
                        const float *cosT, const float *sinT, int max_seq, cudaStream_t s)
{
    smc_dense_out o{};
    o.y = b.qa, o.ldy = d.heads * d.kv_rank;
    int rc = smc_launch_dense_grouped(ctx, b.q, d.heads * (d.dim + d.rot_dim), d.dim + d.rot_dim, b.w_ukt, d.heads, d.kv_rank, d.dim, rw.n, o, s);
    if (rc) return rc;
    const size_t smem = decode_smem(d);
    // as many CTAs per row as keep the device full, up to the cluster limit and to one key tile each
    int cl = DCL;
    const int groups = (d.heads + 15) / 16, most = ((d.window > 0 ? d.window : max_seq) + DT - 1) / DT;
    while (cl > 1 && ((long long)rw.n * groups * cl > ctx->sm_count || cl / 2 >= most)) cl /= 2;
    auto go = [&](auto kernel) {
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        smc_launch_dep_cluster(ctx->use_pdl, cl, kernel, dim3(cl, groups, rw.n), dim3(DTH), smem, s, (const float *)b.qa, (const bf16 *)b.q,
                               (const bf16 *)b.cache, (bf16 *)b.oc, rw, sink, cosT, sinT, d.heads, d.dim, d.kv_rank, d.rot_dim, d.ring, d.window, d.scale,
                               max_seq);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    rc = d.kv_rank <= 256 ? go(latent_decode_kernel<1>) : go(latent_decode_kernel<2>);
    if (rc) return rc;
    o.y = b.o, o.ldy = d.heads * d.vdim, o.y_bf16 = 1;
    const bf16 *wuv = reinterpret_cast<const bf16 *>(w_ukv->d_raw) + (size_t)d.heads * d.dim * d.kv_rank;
    return smc_launch_dense_grouped(ctx, b.oc, d.heads * d.kv_rank, d.kv_rank, wuv, d.heads, d.vdim, d.kv_rank, rw.n, o, s);
}

template <typename T>
int attend_absorbed(smc_ctx *ctx, const smc_latent_dims &d, const smc_latent_bufs &b, const smc_rows &rw, const smc_weight *w_ukv, const float *sink,
                    const float *cosT, const float *sinT, int max_seq, cudaStream_t s)
{
    const bf16 *wuk = reinterpret_cast<const bf16 *>(w_ukv->d_raw), *wuv = wuk + (size_t)d.heads * d.dim * d.kv_rank;
    const int ny = (rw.n + 7) / 8;
    smc_launch_dep(ctx->use_pdl, latent_absorb_kernel<T>, dim3(d.heads, (d.kv_rank + 63) / 64, ny), dim3(256), (size_t)8 * d.dim * sizeof(float), s,
                   static_cast<const T *>(b.q), wuk, b.qa, rw, cosT, sinT, d.heads, d.dim, d.rot_dim, d.kv_rank, max_seq);
    SMC_LAUNCH_CHECK(ctx);
    int rc = attend_rows<T>(ctx, d, b, rw, sink, s);
    if (rc) return rc;
    smc_launch_dep(ctx->use_pdl, latent_value_kernel<T>, dim3((d.heads * d.vdim + 7) / 8, ny), dim3(256), 0, s, static_cast<const float *>(b.oc), wuv,
                   static_cast<T *>(b.o), rw.n, d.heads, d.vdim, d.kv_rank);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

}  // namespace

bool smc_latent_prefill_supported(const smc_latent_dims &d)
{
    return d.dim % 8 == 0 && d.rot_dim % 8 == 0 && d.vdim % 8 == 0 && d.kv_rank % 8 == 0 && d.vdim <= 256 && prefill_smem(d) <= 220 * 1024;
}

bool smc_latent_decode_supported(const smc_latent_dims &d)
{
    return d.dim % 8 == 0 && d.kv_rank % 8 == 0 && d.rot_dim % 8 == 0 && d.kv_rank <= 512 && d.kv_rank + d.rot_dim <= 8 * KPW * 16 && decode_smem(d) <= 220 * 1024;
}

int smc_latent_transpose_uk(smc_ctx *ctx, const smc_latent_dims &d, const smc_weight *w_ukv, void *out, cudaStream_t s)
{
    const size_t n = (size_t)d.heads * d.dim * d.kv_rank;
    transpose_uk_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(reinterpret_cast<const bf16 *>(w_ukv->d_raw), static_cast<bf16 *>(out), d.heads, d.dim,
                                                                   d.kv_rank);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

int smc_latent_check(smc_ctx *ctx, const smc_latent_dims &d)
{
    if (d.kv_rank > 1024) return smc_fail(ctx, SMC_E_UNSUPPORTED, "latent attention: kv_rank %d (up to 1024 are built)", d.kv_rank);
    if (d.rot_dim % 2) return smc_fail(ctx, SMC_E_UNSUPPORTED, "latent attention: an odd rotated part of %d", d.rot_dim);
    if (d.dim > 1024) return smc_fail(ctx, SMC_E_UNSUPPORTED, "latent attention: dim %d (up to 1024 are built)", d.dim);
    return SMC_OK;
}

int smc_latent_post(smc_ctx *ctx, const smc_latent_dims &d, const smc_latent_bufs &b, const smc_rows &rw, int is_bf16, const float *q_norm,
                    const float *kv_norm, const float *cosT, const float *sinT, int max_seq, cudaStream_t s)
{
    auto go = [&](auto *tag) {
        using T = std::remove_pointer_t<decltype(tag)>;
        smc_launch_dep(ctx->use_pdl, latent_post_kernel<T>, dim3((2 * rw.n + 7) / 8), dim3(256), 0, s, static_cast<const T *>(b.down),
                       static_cast<T *>(b.cq), static_cast<T *>(b.cache), rw, q_norm, kv_norm, cosT, sinT, d.q_rank, d.kv_rank, d.rot_dim, d.ring,
                       max_seq, d.eps);
    };
    if (is_bf16) go((bf16 *)nullptr);
    else go((float *)nullptr);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

int smc_latent_attend(smc_ctx *ctx, const smc_latent_dims &d, const smc_latent_bufs &b, const smc_rows &rw, int is_bf16, const smc_weight *w_ukv,
                      const float *sink, const float *cosT, const float *sinT, int max_seq, int pos0, cudaStream_t s)
{
    if (!is_bf16) return attend_absorbed<float>(ctx, d, b, rw, w_ukv, sink, cosT, sinT, max_seq, s);
    if (rw.seq0 < 0 || rw.n < EXPAND_ROWS || !smc_latent_prefill_supported(d)) {
        if (b.w_ukt && smc_latent_decode_supported(d)) return attend_absorbed_mma(ctx, d, b, rw, w_ukv, sink, cosT, sinT, max_seq, s);
        return attend_absorbed<bf16>(ctx, d, b, rw, w_ukv, sink, cosT, sinT, max_seq, s);
    }
    // expanded: the visible rows in order, their keys and values per head, then the tensor cores
    const int k0 = d.window > 0 && pos0 > d.window - 1 ? pos0 - d.window + 1 : 0, nk = pos0 + rw.n - k0, row = d.kv_rank + d.rot_dim;
    const int row16 = row / 8;
    smc_launch_dep(ctx->use_pdl, latent_gather_kernel, dim3((unsigned)(((long long)nk * row16 + 255) / 256)), dim3(256), 0, s,
                   static_cast<const uint4 *>(b.cache), static_cast<uint4 *>(b.keys), rw.seq0, k0, nk, d.ring, row16);
    SMC_LAUNCH_CHECK(ctx);
    smc_dense_out o{};
    o.y = b.kv, o.ldy = d.heads * (d.dim + d.vdim), o.y_bf16 = 1;
    int rc = smc_launch_dense(ctx, b.keys, 1, row, w_ukv, nk, o, s);
    if (rc) return rc;
    const size_t smem = prefill_smem(d);
#define SMC_PREFILL(V)                                                                                                                        \
    do {                                                                                                                                      \
        SMC_CUDA(ctx, cudaFuncSetAttribute(latent_prefill_kernel<V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));                \
        smc_launch_dep(ctx->use_pdl, latent_prefill_kernel<V>, dim3(d.heads, (rw.n + 63) / 64), dim3(128), smem, s, (const bf16 *)b.q,        \
                       (const bf16 *)b.keys, (const bf16 *)b.kv, (bf16 *)b.o, sink, cosT, sinT, rw.n, nk, pos0, k0, d.heads, d.dim,           \
                       d.rot_dim, d.vdim, d.kv_rank, d.window, d.scale, max_seq);                                                             \
    } while (0)
    if (d.vdim <= 32) SMC_PREFILL(4);
    else if (d.vdim <= 64) SMC_PREFILL(8);
    else if (d.vdim <= 128) SMC_PREFILL(16);
    else SMC_PREFILL(32);
#undef SMC_PREFILL
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

// ------------------------------------------------------------------------------ tables
// Angles p * f_i in double on the host, cosine and sine rounded to fp32.
extern "C" int smc_rope_tables_yarn(smc_ctx *ctx, const smc_rotation *rot, int maxSeq, float *d_cos, float *d_sin)
{
    if (!ctx || !rot || !d_cos || !d_sin || rot->dims <= 0 || rot->dims % 2 || maxSeq <= 0 || !(rot->base > 0))
        return smc_fail(ctx, SMC_E_INVALID, "rope_tables_yarn: bad arguments");
    const int half = rot->dims / 2;
    std::vector<double> f(half);
    for (int i = 0; i < half; ++i) f[i] = pow(rot->base, -2.0 * i / rot->dims);
    double factor = 1.0;
    if (rot->factor > 0) {
        auto turns_at = [&](double turns) { return rot->dims * log(rot->original / (2.0 * M_PI * turns)) / (2.0 * log(rot->base)); };
        const double lo = fmax(floor(turns_at(rot->fast)), 0.0), hi = fmin(ceil(turns_at(rot->slow)), rot->dims - 1.0);
        for (int i = 0; i < half; ++i) {
            const double r = fmin(fmax((i - lo) / fmax(hi - lo, 0.001), 0.0), 1.0);
            f[i] = f[i] / rot->factor * r + f[i] * (1.0 - r);
        }
        factor = 0.1 * log(rot->factor) + 1.0;
    }
    std::vector<float> c((size_t)maxSeq * half), s((size_t)maxSeq * half);
    for (int p = 0; p < maxSeq; ++p)
        for (int i = 0; i < half; ++i) {
            const double a = p * f[i];
            c[(size_t)p * half + i] = (float)(cos(a) * factor), s[(size_t)p * half + i] = (float)(sin(a) * factor);
        }
    SMC_CUDA(ctx, cudaMemcpy(d_cos, c.data(), c.size() * sizeof(float), cudaMemcpyHostToDevice));
    SMC_CUDA(ctx, cudaMemcpy(d_sin, s.data(), s.size() * sizeof(float), cudaMemcpyHostToDevice));
    return SMC_OK;
}
