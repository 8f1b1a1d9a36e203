// Attention heads over a sliding window: grouped key/value heads, an optional RMS norm of queries and keys per head, an
// optional learned bias per distance and head, softmax over the keys seen.
//   score(i, j) = (q_i . k_j) scale + bias[h][i - j],  0 <= i - j < window
// The cache is a ring: position p lives in row p % ring, ring >= window - 1 + the longest portion, so the rows a portion
// writes never displace one that its first query still sees.  A row holds key and value of each key/value head side by side.
//
//   attn_decode_kernel    bfloat16, one row per sequence: norms, cache append and attention in one launch, the window's keys
//                         dealt to the warps of a cluster of CTAs
//   attn_prefill_kernel   bfloat16, portions: 64 query rows of a head per CTA
//   attn_post_kernel      norms and cache append for the forms that do not do it themselves
//   attn_rows_kernel      fp32 and odd sizes
#include <math.h>

#include <type_traits>
#include <vector>

#include "smc_mma.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

// dst = RMSNorm(src) * w of one head by one warp (w null: a copy), V elements at a time; dst2 (may be null) gets the same
template <typename T, int V>
__device__ __forceinline__ void head_norm(const T *src, const float *w, int n, float eps, T *dst, T *dst2 = nullptr)
{
    const int lane = threadIdx.x & 31;
    float inv = 1.0f, v[V], g[V];
    if (w) {
        float ss = 0.f;
        for (int i = lane * V; i < n; i += 32 * V) {
            load_v<T, V>(src + i, v);
#pragma unroll
            for (int j = 0; j < V; ++j) ss = fmaf(v[j], v[j], ss);
        }
        inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(smc_group_sum<32>(ss), (float)n) + eps));
    }
    for (int i = lane * V; i < n; i += 32 * V) {
        load_v<T, V>(src + i, v);
        if (w) {
            load_v<float, V>(w + i, g);
#pragma unroll
            for (int j = 0; j < V; ++j) v[j] = (v[j] * inv) * g[j];
        }
        store_v<T, V>(dst + i, v);
        if (dst2) store_v<T, V>(dst2 + i, v);
    }
}

// A warp per (row, head): queries into q, keys and values into the cache.
template <typename T, int V>
__global__ void __launch_bounds__(256) attn_post_kernel(const T *__restrict__ in, int ld, int col, T *__restrict__ q, T *__restrict__ cache, smc_rows rw,
                                                        const float *__restrict__ qn, const float *__restrict__ kn, int heads, int kvh, int dim,
                                                        int vdim, int ring, float eps)
{
    smc_grid_dep_sync();
    const int units = heads + 2 * kvh;
    const long long wid = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int r = (int)(wid / units), u = (int)(wid % units);
    if (r >= rw.n) return;
    const T *src = in + (size_t)r * ld + col;
    if (u < heads) return head_norm<T, V>(src + u * dim, qn, dim, eps, q + ((size_t)r * heads + u) * dim);
    int slot, p;
    row_place(rw, r, slot, p);
    const int k = (u - heads) % kvh;
    T *dst = cache + (((size_t)slot * ring + p % ring) * kvh + k) * (dim + vdim);
    if (u < heads + kvh) head_norm<T, V>(src + (size_t)(heads + k) * dim, kn, dim, eps, dst);
    else head_norm<T, V>(src + (size_t)(heads + kvh) * dim + k * vdim, nullptr, vdim, eps, dst + dim);
}

// The same for bfloat16 heads of up to 128 elements in whole eights: half a warp per head, eight heads of a row per warp.
__global__ void __launch_bounds__(256) attn_post8_kernel(const bf16 *__restrict__ in, int ld, int col, bf16 *__restrict__ q, bf16 *__restrict__ cache,
                                                         smc_rows rw, const float *__restrict__ qn, const float *__restrict__ kn, int heads, int kvh,
                                                         int dim, int vdim, int ring, float eps)
{
    const int units = heads + 2 * kvh, per = (units + 7) / 8, sub = threadIdx.x >> 4 & 1, i = 8 * (threadIdx.x & 15);
    float g[2][8];  // the weights of queries and keys
#pragma unroll
    for (int k = 0; k < 8; ++k) g[0][k] = qn && i + k < dim ? qn[i + k] : 1.f, g[1][k] = kn && i + k < dim ? kn[i + k] : 1.f;
    smc_grid_dep_sync();
    const int wid = blockIdx.x * 8 + (threadIdx.x >> 5), r = wid / per, u0 = wid % per * 8 + sub;
    if (r >= rw.n) return;
    int slot, p;
    row_place(rw, r, slot, p);
    const bf16 *src = in + (size_t)r * ld + col;
    bf16 *row = cache + ((size_t)slot * ring + p % ring) * kvh * (dim + vdim);
    uint4 raw[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int u = u0 + 2 * j, v = u - heads - kvh;
        raw[j] = make_uint4(0u, 0u, 0u, 0u);
        if (u < units && i < (v < 0 ? dim : vdim)) raw[j] = *reinterpret_cast<const uint4 *>(v < 0 ? src + u * dim + i : src + (heads + kvh) * dim + v * vdim + i);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int u = u0 + 2 * j, v = u - heads - kvh;
        const bool key = u >= heads;
        const bf16 *e = reinterpret_cast<const bf16 *>(&raw[j]);
        float x[8], ss = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) x[k] = to_f(e[k]), ss = fmaf(x[k], x[k], ss);
#pragma unroll
        for (int d = 1; d < 16; d <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
        if (v < 0 && (key ? kn : qn)) {
            const float inv = rsqrtf(__fdividef(ss, (float)dim) + eps);
#pragma unroll
            for (int k = 0; k < 8; ++k) x[k] = (x[k] * inv) * (key ? g[1][k] : g[0][k]);
            raw[j] = make_uint4(pack2(x[0], x[1]), pack2(x[2], x[3]), pack2(x[4], x[5]), pack2(x[6], x[7]));
        }
        bf16 *dst = !key ? q + ((size_t)r * heads + u) * dim : (v < 0 ? row + (u - heads) * (dim + vdim) : row + v * (dim + vdim) + dim);
        if (u < units && i < (v < 0 ? dim : vdim)) *reinterpret_cast<uint4 *>(dst + i) = raw[j];
    }
}

// One CTA per (head, row); the warps take every eighth key with a running maximum each and are merged at the end.
template <typename T, int EPL>
__global__ void __launch_bounds__(256) attn_rows_kernel(const T *__restrict__ q, const T *__restrict__ cache, T *__restrict__ out, int ldo, smc_rows rw,
                                                        const float *__restrict__ bias, int bias_len, int heads, int kvh, int dim, int vdim, int ring,
                                                        int window, float scale, float out_scale)
{
    extern __shared__ float sm[];  // query [dim], then partial sums [8][vdim]
    __shared__ float sm_m[8], sm_l[8];
    smc_grid_dep_sync();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.x, r = blockIdx.y, row = dim + vdim;
    float *qs = sm, *part = sm + dim;
    for (int i = threadIdx.x; i < dim; i += 256) qs[i] = to_f(q[((size_t)r * heads + h) * dim + i]);
    __syncthreads();
    int slot, p;
    row_place(rw, r, slot, p);
    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    const T *base = cache + ((size_t)slot * ring * kvh + h / (heads / kvh)) * row;
    float o[EPL], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int j = 0; j < EPL; ++j) o[j] = 0.f;
    for (int k = lo + warp; k <= p; k += 8) {
        const T *kr = base + (size_t)(k % ring) * kvh * row;
        float s = 0.f;
        for (int i = lane; i < dim; i += 32) s = fmaf(qs[i], to_f(kr[i]), s);
        s = smc_group_sum<32>(s) * scale;
        if (bias) s += bias[(size_t)h * bias_len + min(p - k, bias_len - 1)];
        const float nm = fmaxf(m, s), f = expf(m - nm), e = expf(s - nm);
        l = fmaf(l, f, e), m = nm;
#pragma unroll
        for (int j = 0; j < EPL; ++j)
            if (lane + 32 * j < vdim) o[j] = fmaf(e, to_f(kr[dim + lane + 32 * j]), o[j] * f);
    }
#pragma unroll
    for (int j = 0; j < EPL; ++j)
        if (lane + 32 * j < vdim) part[warp * vdim + lane + 32 * j] = o[j];
    if (lane == 0) sm_m[warp] = m, sm_l[warp] = l;
    __syncthreads();
    float top = -INFINITY;
#pragma unroll
    for (int w = 0; w < 8; ++w) top = fmaxf(top, sm_m[w]);
    float f[8], den = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) f[w] = expf(sm_m[w] - top), den = fmaf(f[w], sm_l[w], den);
    const float inv = __fdiv_rn(1.0f, den);
    for (int i = threadIdx.x; i < vdim; i += 256) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v = fmaf(f[w], part[w * vdim + i], v);
        out[(size_t)r * ldo + h * vdim + i] = from_f<T>(v * inv * out_scale);
    }
}

// ------------------------------------------------------------------------------ one row per sequence, bfloat16
// Up to 16 query heads that share a key/value head per cluster of up to eight CTAs of four warps.  A warp takes every
// (4 * cluster)-th tile of 16 keys into a three-stage ring of its own (no CTA barrier in the loop), keeps a running
// (maximum, sum) and its part of the weighted values; the parts meet in (distributed) shared memory.  The row's own key is
// normed, stored and put into the last tile by the warp that takes it.  Keys and the position are fetched BEFORE the wait for the
// predecessor: a kernel that is launched early is so only after every CTA of its predecessor has passed its own wait, and
// the older keys and the positions were written before the predecessor's launch.
constexpr int DKT = 16, DST = 3, DWP = 4, DCL = 8;
__host__ __device__ constexpr int tile_ld(int n) { return (((n + 15) & ~15) + 8) * 2; }  // bytes: an odd number of 16-byte units
__host__ __device__ constexpr int decode_smem(int dim, int vdim) { return 16 * tile_ld(dim) + DWP * DST * DKT * (tile_ld(dim) + tile_ld(vdim)) + 2 * (dim + vdim); }

// VT: value tiles of 8 columns; HALF: up to eight heads (the other half of each fragment is not used); QS > 0: the queries'
// fragments (16 elements each, up to QS of them) stay in registers.
template <int VT, bool HALF, int QS>
__global__ void __launch_bounds__(DWP * 32)
attn_decode_kernel(const bf16 *__restrict__ in, int ld, int col, bf16 *cache, bf16 *__restrict__ out, int ldo, smc_rows rw, const float *__restrict__ qn,
                   const float *__restrict__ kn, const float *__restrict__ bias, int bias_len, int heads, int kvh, int dim, int vdim, int ring,
                   int window, float scale, float out_scale, float eps)
{
    extern __shared__ __align__(16) uint8_t sm_raw[];
    __shared__ float w_m[DWP][16], w_l[DWP][16], all_f[DCL * DWP][16];
    const int ldk = tile_ld(dim), ldv = tile_ld(vdim), d16 = (dim + 15) & ~15, row = dim + vdim;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int G = heads / kvh, groups = (G + 15) / 16, kh = blockIdx.y / groups, grp = blockIdx.y % groups;
    const int h0 = kh * G + grp * 16, nh = min(16, G - grp * 16), r = blockIdx.z, rank = blockIdx.x, cl = gridDim.x;
    const int stage = DKT * (ldk + ldv);
    uint8_t *mine = sm_raw + 16 * ldk + warp * DST * stage;
    const uint32_t qb = (uint32_t)__cvta_generic_to_shared(sm_raw), kb0 = (uint32_t)__cvta_generic_to_shared(mine);
    // the query rows without a head, and padding columns that no copy writes
    bf16 *own = reinterpret_cast<bf16 *>(sm_raw + 16 * ldk + DWP * DST * stage);  // the row's own key and value
    const int clear = d16 != dim ? 16 * ldk + DWP * DST * stage : 16 * ldk;
    for (int e = threadIdx.x; e < clear / 16; e += DWP * 32) reinterpret_cast<uint4 *>(sm_raw)[e] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();

    int slot, p;
    row_place(rw, r, slot, p);
    const int old = window > 0 ? min(p, window - 1) : p, lo_row = (p - old) % ring, tiles = old / DKT + 1;
    bf16 *base = cache + ((size_t)slot * ring * kvh + kh) * row;
    const int cu = dim / 8, pieces = row / 8, step = cl * DWP;
    const size_t pitch = (size_t)kvh * row;
    auto fetch = [&](int t, int st) {
        if (t < tiles) {
            const uint32_t kb = kb0 + (uint32_t)(st * stage);
            int first = lo_row + t * DKT;
            first -= first >= ring ? ring : 0;  // old < ring
            const bool straight = (t + 1) * DKT <= old && first + DKT <= ring;
            for (int c = lane; c < pieces; c += 32) {
                uint32_t dst = c < cu ? kb + (uint32_t)(16 * c) : kb + (uint32_t)(DKT * ldk + 16 * (c - cu));
                const uint32_t ldd = c < cu ? ldk : ldv;
                const bf16 *src = base + (size_t)first * pitch + 8 * c;
                if (straight) {
#pragma unroll
                    for (int j = 0; j < DKT; ++j, dst += ldd, src += pitch) cp16(dst, src, true);
                } else {
#pragma unroll 1
                    for (int j = 0; j < DKT; ++j, dst += ldd) {
                        const bool seen = t * DKT + j < old;
                        const int rr = first + j - (first + j >= ring ? ring : 0);
                        cp16(dst, seen ? base + (size_t)rr * pitch + 8 * c : base, seen);
                    }
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    int t = warp * cl + rank;
    fetch(t, 0), fetch(t + step, 1);
    smc_grid_dep_sync();
    const bf16 *src = in + (size_t)r * ld + col;
    for (int hh = warp; hh < nh; hh += DWP)
        head_norm<bf16, 4>(src + (size_t)(h0 + hh) * dim, qn, dim, eps, reinterpret_cast<bf16 *>(sm_raw + hh * ldk));
    const bool last = (tiles - 1) % step == warp * cl + rank;  // this warp takes the last tile
    if (last) {
        bf16 *keep = base + (size_t)(p % ring) * kvh * row;
        head_norm<bf16, 4>(src + (size_t)(heads + kh) * dim, kn, dim, eps, own, grp == 0 ? keep : nullptr);
        head_norm<bf16, 4>(src + (size_t)(heads + kvh) * dim + kh * vdim, nullptr, vdim, eps, own + dim, grp == 0 ? keep + dim : nullptr);
    }
    __syncthreads();

    float o[VT][4], m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
#pragma unroll
    for (int n = 0; n < VT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const float scale2 = scale * LOG2E;
    const float *b0 = bias && g < nh ? bias + (size_t)(h0 + g) * bias_len : nullptr, *b1 = bias && g + 8 < nh ? bias + (size_t)(h0 + g + 8) * bias_len : nullptr;
    const uint32_t a_off = qb + (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + 16 * (lane >> 4));
    const uint32_t k_off = (uint32_t)(((lane & 7) + 8 * (lane >> 4)) * ldk + 16 * ((lane >> 3) & 1));
    const uint32_t v_off = (uint32_t)(DKT * ldk + ((lane & 7) + 8 * ((lane >> 3) & 1)) * ldv + 16 * (lane >> 4));
    constexpr int R = HALF ? 1 : 2;  // fragment rows in use per lane
    uint32_t aq[QS ? QS : 1][4];
#pragma unroll
    for (int ks = 0; ks < QS; ++ks) {
        aq[ks][0] = aq[ks][1] = aq[ks][2] = aq[ks][3] = 0u;
        if (ks < d16 / 16) ldsm4(a_off + 32 * ks, aq[ks]);
    }
    // a tile whose first n keys count, key j at distance d - j
    auto take = [&](uint32_t tile, int n, int d) {
        float c[R][4];
#pragma unroll
        for (int h = 0; h < R; ++h)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float *bh = h ? b1 : b0;
                c[h][i] = bh ? __ldg(bh + max(0, d - (8 * (i >> 1) + 2 * tg + (i & 1)))) : 0.f;  // (d < bias_len)
            }
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
        auto part = [&](const uint32_t (&a)[4], int ks) {
            uint32_t b[4];
            ldsm4(tile + k_off + 32 * ks, b);
            mma_bf16(s[0], a, b[0], b[1]);
            mma_bf16(s[1], a, b[2], b[3]);
        };
        if (QS) {
#pragma unroll
            for (int ks = 0; ks < QS; ++ks)
                if (ks < d16 / 16) part(aq[ks], ks);
        } else {
#pragma unroll 4
            for (int ks = 0; ks < d16 / 16; ++ks) {
                uint32_t a[4];
                ldsm4(a_off + 32 * ks, a);
                part(a, ks);
            }
        }
        float f[2] = {1.f, 1.f}, e[2][4] = {};
#pragma unroll
        for (int h = 0; h < R; ++h) {
            float top = -INFINITY;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                e[h][i] = fmaf(s[i >> 1][2 * h + (i & 1)], scale2, c[h][i] * LOG2E);
                if (n < DKT) e[h][i] = 8 * (i >> 1) + 2 * tg + (i & 1) < n ? e[h][i] : -INFINITY;
                top = fmaxf(top, e[h][i]);
            }
            top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1)), top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
            float &m = h ? m1 : m0, &l = h ? l1 : l0;
            top = fmaxf(m, top);  // finite: the first key of a tile always counts
            f[h] = ex2(m - top), m = top;
#pragma unroll
            for (int i = 0; i < 4; ++i) e[h][i] = ex2(e[h][i] - top);
            l = fmaf(l, f[h], (e[h][0] + e[h][1]) + (e[h][2] + e[h][3]));
        }
        const uint32_t w[4] = {pack2(e[0][0], e[0][1]), HALF ? 0u : pack2(e[1][0], e[1][1]), pack2(e[0][2], e[0][3]), HALF ? 0u : pack2(e[1][2], e[1][3])};
        if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
            for (int i = 0; i < VT; ++i) {
                o[i][0] *= f[0], o[i][1] *= f[0];
                if (!HALF) o[i][2] *= f[1], o[i][3] *= f[1];
            }
        }
#pragma unroll
        for (int i = 0; i < VT / 2; ++i)
            if (16 * i < vdim) {
                uint32_t b[4];
                ldsm4t(tile + v_off + 32 * i, b);
                mma_bf16(o[2 * i], w, b[0], b[1]);
                mma_bf16(o[2 * i + 1], w, b[2], b[3]);
            }
    };
    int st = 0;
    for (; t < tiles; t += step) {
        fetch(t + 2 * step, st == 0 ? 2 : st - 1);
        asm volatile("cp.async.wait_group 2;" ::: "memory");
        __syncwarp();
        if (last && t == tiles - 1) {
            uint8_t *kr = mine + st * stage + (old % DKT) * ldk, *vr = mine + st * stage + DKT * ldk + (old % DKT) * ldv;
            for (int c = lane; c < pieces; c += 32)
                *reinterpret_cast<uint4 *>(c < cu ? kr + 16 * c : vr + 16 * (c - cu)) = *reinterpret_cast<const uint4 *>(own + 8 * c);
            __syncwarp();
        }
        take(kb0 + (uint32_t)(st * stage), min(DKT, old + 1 - t * DKT), old - t * DKT);
        __syncwarp();  // the stage is refilled by the next iteration's fetch
        st = st == 2 ? 0 : st + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
    // ---- the parts: [16][vdim] fp32 over each warp's own tiles
    const int ldp = ((vdim + 15) & ~15) + 4;
    float *part = reinterpret_cast<float *>(mine);
#pragma unroll
    for (int n = 0; n < VT; ++n) {
        const int c = 8 * n + 2 * tg;
        if (c >= vdim) continue;
        *reinterpret_cast<float2 *>(part + g * ldp + c) = make_float2(o[n][0], o[n][1]);
        if (!HALF) *reinterpret_cast<float2 *>(part + (g + 8) * ldp + c) = make_float2(o[n][2], o[n][3]);
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1), l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1), l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (tg == 0) w_m[warp][g] = m0, w_m[warp][g + 8] = m1, w_l[warp][g] = l0, w_l[warp][g + 8] = l1;
    auto cluster_sync = [] { asm volatile("barrier.cluster.arrive;\n\tbarrier.cluster.wait;" ::: "memory"); };
    cluster_sync();
    auto remote = [](const void *ptr, int cta) {
        uint32_t a = (uint32_t)__cvta_generic_to_shared(ptr), v;
        float f;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(v) : "r"(a), "r"(cta));
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(f) : "r"(v) : "memory");
        return f;
    };
    {  // factors: eight lanes per head, each with every eighth part
        const int hh = threadIdx.x >> 3, sub = threadIdx.x & 7, parts = cl * DWP;
        float m[DCL * DWP / 8], l[DCL * DWP / 8], top = -INFINITY, den = 0.f;
#pragma unroll
        for (int i = 0; i < DCL * DWP / 8; ++i) {
            const int k = sub + 8 * i;
            m[i] = k < parts ? remote(&w_m[k % DWP][hh], k / DWP) : -INFINITY, l[i] = k < parts ? remote(&w_l[k % DWP][hh], k / DWP) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < DCL * DWP / 8; ++i) top = fmaxf(top, m[i]);
#pragma unroll
        for (int x = 1; x < 8; x <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, x));
#pragma unroll
        for (int i = 0; i < DCL * DWP / 8; ++i) m[i] = ex2(m[i] - top), den = fmaf(m[i], l[i], den);  // a warp without a key: 0
#pragma unroll
        for (int x = 1; x < 8; x <<= 1) den += __shfl_xor_sync(0xffffffffu, den, x);
        const float inv = __fdiv_rn(out_scale, den);
#pragma unroll
        for (int i = 0; i < DCL * DWP / 8; ++i) all_f[sub + 8 * i][hh] = m[i] * inv;
    }
    __syncthreads();
    const int total = nh * vdim, per = (total + cl - 1) / cl, e1 = min(total, (rank + 1) * per);
    const int region = DST * stage / 4;  // floats between the warps' parts
    const float *part0 = reinterpret_cast<const float *>(sm_raw + 16 * ldk);
    for (int e = rank * per + threadIdx.x; e < e1; e += DWP * 32) {
        const int hh = e / vdim, c = e % vdim;
        float v = 0.f, x[DCL][DWP];
#pragma unroll
        for (int k = 0; k < DCL; ++k)
#pragma unroll
            for (int w = 0; w < DWP; ++w) x[k][w] = k < cl ? remote(part0 + (size_t)w * region + hh * ldp + c, k) : 0.f;
#pragma unroll
        for (int k = 0; k < DCL; ++k)
#pragma unroll
            for (int w = 0; w < DWP; ++w) v = fmaf(all_f[k * DWP + w][hh], x[k][w], v);
        out[(size_t)r * ldo + (size_t)(h0 + hh) * vdim + c] = __float2bfloat16_rn(v);
    }
    cluster_sync();  // nobody leaves while its parts are read
}

// ------------------------------------------------------------------------------ portions, bfloat16
// 64 query rows of one head per CTA (16 per warp), key tiles of 64 from the ring, two tile buffers filled by cp.async.
// Scores, biases and the running softmax are fp32; the weights enter the second product as bfloat16.  Head sizes are padded
// to 16 with zeros in shared memory.  VT: value tiles of 8 columns a thread keeps accumulators for.
constexpr int PQ = 64, PK = 64;
__host__ __device__ constexpr int prefill_smem(int dim, int vdim) { return PQ * tile_ld(dim) + 2 * PK * (tile_ld(dim) + tile_ld(vdim)) + 2 * (PQ + PK) * 4; }

template <int VT>
__global__ void __launch_bounds__(128)
attn_prefill_kernel(const bf16 *__restrict__ q, const bf16 *__restrict__ cache, bf16 *__restrict__ out, int ldo, const float *__restrict__ bias,
                    int bias_len, int T, int slot, int pos0, int heads, int kvh, int dim, int vdim, int ring, int window, float scale, float out_scale)
{
    extern __shared__ __align__(16) uint8_t sm_raw[];
    const int ldk = tile_ld(dim), ldv = tile_ld(vdim), d16 = (dim + 15) & ~15, v16 = (vdim + 15) & ~15, row = dim + vdim;
    const uint32_t sq = (uint32_t)__cvta_generic_to_shared(sm_raw), sk = sq + PQ * ldk, sv = sk + 2 * PK * ldk;
    float *sb = reinterpret_cast<float *>(sm_raw + PQ * ldk + 2 * PK * (ldk + ldv));  // two tiles' biases by query - key
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tg = lane & 3;
    const int h = blockIdx.x, kh = h / (heads / kvh), t0 = (int)(gridDim.y - 1 - blockIdx.y) * PQ;
    // padding columns are never written by the copies below: clear everything once
    for (uint32_t e = threadIdx.x; e < (uint32_t)prefill_smem(dim, vdim) / 16; e += 128) reinterpret_cast<uint4 *>(sm_raw)[e] = make_uint4(0u, 0u, 0u, 0u);
    smc_grid_dep_sync();
    __syncthreads();

    const int p_first = pos0 + t0, p_last = pos0 + min(T, t0 + PQ) - 1;  // positions of the CTA's queries
    const int key_lo = window > 0 ? max(0, p_first - window + 1) : 0;     // positions of its keys, both ends included
    const int key_hi = p_last, lo_row = key_lo % ring;
    const bf16 *base = cache + ((size_t)slot * ring * kvh + kh) * row;
    const size_t pitch = (size_t)kvh * row;
    // columns of the ring's rows -> tile, 16 bytes per thread and copy; keys past the last visible one become zeros
    auto copy = [&](uint32_t dst, int ldd, const bf16 *src, int pieces, int start) {
        const int c0 = threadIdx.x & 15, j0 = threadIdx.x >> 4, first = lo_row + (start - key_lo);
        for (int c = c0; c < pieces; c += 16) {
#pragma unroll 4
            for (int j = j0; j < PK; j += 8) {
                const bool in = start + j <= key_hi;
                int rr = first + j;
                rr -= rr >= ring ? ring : 0;  // the visible keys fit the ring
                cp16(dst + (uint32_t)(j * ldd + 16 * c), in ? src + (size_t)rr * pitch + 8 * c : src, in);
            }
        }
    };
    auto fetch = [&](int start, int buf) {
        copy(sk + (uint32_t)(buf * PK * ldk), ldk, base, dim / 8, start);
        copy(sv + (uint32_t)(buf * PK * ldv), ldv, base + dim, vdim / 8, start);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (bias) {
            const int d = p_first - (start + PK - 1) + (int)threadIdx.x;
            sb[buf * (PQ + PK) + threadIdx.x] = bias[(size_t)h * bias_len + max(0, min(d, bias_len - 1))] * LOG2E;
        }
    };
    fetch(key_lo, 0);
    const int cu = dim / 8;
    for (int e = threadIdx.x; e < PQ * cu; e += 128) {
        const int r = e / cu, c = e % cu;
        if (t0 + r < T)
            *reinterpret_cast<uint4 *>(sm_raw + r * ldk + 16 * c) = *reinterpret_cast<const uint4 *>(q + ((size_t)(t0 + r) * heads + h) * dim + 8 * c);
    }
    const int tile_hi = p_first, tile_lo = window > 0 ? p_first + PQ - window : 0;  // keys all of the CTA's queries see
    const int r0 = warp * 16 + g, r1 = r0 + 8;                                      // the thread's two rows; the keys each sees
    int hi0 = -1, hi1 = -1, lo0 = 0, lo1 = 0;
    if (t0 + r0 < T) hi0 = p_first + r0, lo0 = window > 0 ? max(0, hi0 - window + 1) : 0;
    if (t0 + r1 < T) hi1 = p_first + r1, lo1 = window > 0 ? max(0, hi1 - window + 1) : 0;
    const float scale2 = scale * LOG2E;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    float o[VT][4];
#pragma unroll
    for (int n = 0; n < VT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const uint32_t a_off = sq + (uint32_t)((warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ldk + 16 * (lane >> 4));
    const uint32_t bk_off = (uint32_t)(((lane & 7) + 8 * (lane >> 4)) * ldk + 16 * ((lane >> 3) & 1));
    const uint32_t bv_off = (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * ldv + 16 * (lane >> 4));

    int buf = 0;
    for (int start = key_lo; start <= key_hi; start += PK, buf ^= 1) {
        if (start + PK <= key_hi) {
            fetch(start + PK, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t kb = sk + (uint32_t)(buf * PK * ldk) + bk_off, vb = sv + (uint32_t)(buf * PK * ldv) + bv_off;
        float s[PK / 8][4];
#pragma unroll
        for (int n = 0; n < PK / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll 4
        for (int ks = 0; ks < d16 / 16; ++ks) {
            uint32_t a[4];
            ldsm4(a_off + 32 * ks, a);
#pragma unroll
            for (int np = 0; np < PK / 16; ++np) {
                uint32_t b[4];
                ldsm4(kb + np * 16 * ldk + 32 * ks, b);
                mma_bf16(s[2 * np], a, b[0], b[1]);
                mma_bf16(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        // biases of (row r, key j) at r - j + PK - 1; zeros without a bias
        const float *bt = sb + buf * (PQ + PK) + r0 + PK - 1 - 2 * tg;
        float tm0 = -INFINITY, tm1 = -INFINITY;
        const bool whole = start >= tile_lo && start + PK - 1 <= tile_hi;  // every query of the CTA sees the whole tile
#pragma unroll
        for (int n = 0; n < PK / 8; ++n) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int key = start + 8 * n + 2 * tg + i;
                s[n][i] = fmaf(s[n][i], scale2, bt[-8 * n - i]), s[n][2 + i] = fmaf(s[n][2 + i], scale2, bt[8 - 8 * n - i]);
                if (!whole) {
                    s[n][i] = key >= lo0 && key <= hi0 ? s[n][i] : -INFINITY;
                    s[n][2 + i] = key >= lo1 && key <= hi1 ? s[n][2 + i] : -INFINITY;
                }
                tm0 = fmaxf(tm0, s[n][i]), tm1 = fmaxf(tm1, s[n][2 + i]);
            }
        }
        tm0 = fmaxf(tm0, __shfl_xor_sync(0xffffffffu, tm0, 1)), tm0 = fmaxf(tm0, __shfl_xor_sync(0xffffffffu, tm0, 2));
        tm1 = fmaxf(tm1, __shfl_xor_sync(0xffffffffu, tm1, 1)), tm1 = fmaxf(tm1, __shfl_xor_sync(0xffffffffu, tm1, 2));
        const float nm0 = fmaxf(m0, tm0), nm1 = fmaxf(m1, tm1);
        // a row that has seen nothing yet keeps maximum -inf; its weights are 0
        const float b0 = nm0 > -INFINITY ? nm0 : 0.f, b1 = nm1 > -INFINITY ? nm1 : 0.f;
        const float c0 = ex2(m0 - b0), c1 = ex2(m1 - b1);
        float ps0 = 0.f, ps1 = 0.f;
        uint32_t p[PK / 16][4];
#pragma unroll
        for (int n = 0; n < PK / 8; ++n) {
            const float e0 = ex2(s[n][0] - b0), e1 = ex2(s[n][1] - b0), e2 = ex2(s[n][2] - b1), e3 = ex2(s[n][3] - b1);
            ps0 += e0 + e1, ps1 += e2 + e3;
            p[n >> 1][(n & 1) * 2] = pack2(e0, e1), p[n >> 1][(n & 1) * 2 + 1] = pack2(e2, e3);
        }
        l0 = fmaf(l0, c0, ps0), l1 = fmaf(l1, c1, ps1);  // a lane's own columns; summed over the row's lanes at the end
        m0 = nm0, m1 = nm1;
#pragma unroll
        for (int n = 0; n < VT; ++n) o[n][0] *= c0, o[n][1] *= c0, o[n][2] *= c1, o[n][3] *= c1;
#pragma unroll
        for (int j = 0; j < PK / 16; ++j)
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
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1), l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1), l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    const float i0 = l0 > 0.f ? __fdiv_rn(out_scale, l0) : 0.f, i1 = l1 > 0.f ? __fdiv_rn(out_scale, l1) : 0.f;
#pragma unroll
    for (int n = 0; n < VT; ++n) {
        const int c = 8 * n + 2 * tg;
        if (c >= vdim) continue;
        if (t0 + r0 < T) *reinterpret_cast<uint32_t *>(out + (size_t)(t0 + r0) * ldo + h * vdim + c) = pack2(o[n][0] * i0, o[n][1] * i0);
        if (t0 + r1 < T) *reinterpret_cast<uint32_t *>(out + (size_t)(t0 + r1) * ldo + h * vdim + c) = pack2(o[n][2] * i1, o[n][3] * i1);
    }
}

__global__ void __launch_bounds__(256) expand_bias_kernel(const float *__restrict__ table, const int *__restrict__ bucket, int heads, int len,
                                                          float *__restrict__ out)
{
    const long long e = (long long)blockIdx.x * 256 + threadIdx.x;
    if (e < (long long)heads * len) out[e] = table[(size_t)bucket[e % len] * heads + e / len];
}

bool whole(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
// rows and 16-byte pieces that the tensor-core kernels can copy
bool pieces_fit(const smc_attn_dims &d, const smc_attn_bufs &b)
{
    return d.dim % 8 == 0 && d.vdim % 8 == 0 && d.vdim <= 256 && b.ld % 2 == 0 && b.ldo % 2 == 0 && whole(b.q) && whole(b.cache) &&
           (reinterpret_cast<uintptr_t>(b.o) & 3) == 0;
}

template <typename F>
int by_value_tiles(int vdim, F go)
{
    if (vdim <= 64) return go(std::integral_constant<int, 8>());
    if (vdim <= 128) return go(std::integral_constant<int, 16>());
    return go(std::integral_constant<int, 32>());
}

template <typename T>
int post(smc_ctx *ctx, const smc_attn_dims &d, const smc_attn_bufs &b, const smc_rows &rw, cudaStream_t s)
{
    auto go = [&](auto kernel, int units) {
        const long long warps = (long long)rw.n * units;
        smc_launch_dep(ctx->use_pdl, kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, s, static_cast<const T *>(b.in), b.ld, b.col,
                       static_cast<T *>(b.q), static_cast<T *>(b.cache), rw, b.q_norm, b.k_norm, d.heads, d.kv_heads, d.dim, d.vdim, d.ring, d.eps);
    };
    const bool four = d.dim % 4 == 0 && d.vdim % 4 == 0 && b.ld % 4 == 0 && b.col % 4 == 0 && whole(b.in) && whole(b.q) && whole(b.cache) &&
                      whole(b.q_norm) && whole(b.k_norm);
    const int units = d.heads + 2 * d.kv_heads;
    if constexpr (std::is_same<T, bf16>::value)
        if (four && d.dim <= 128 && d.vdim <= 128 && d.dim % 8 == 0 && d.vdim % 8 == 0 && b.ld % 8 == 0 && b.col % 8 == 0) {
            go(attn_post8_kernel, (units + 7) / 8);
            SMC_LAUNCH_CHECK(ctx);
            return SMC_OK;
        }
    four ? go(attn_post_kernel<T, 4>, units) : go(attn_post_kernel<T, 1>, units);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

template <typename T>
int rows(smc_ctx *ctx, const smc_attn_dims &d, const smc_attn_bufs &b, const smc_rows &rw, cudaStream_t s)
{
    int rc = post<T>(ctx, d, b, rw, s);
    if (rc) return rc;
    const size_t smem = ((size_t)d.dim + 8 * d.vdim) * sizeof(float);
    auto go = [&](auto kernel) {
        if (smem > 40 * 1024) SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(d.heads, rw.n), dim3(256), smem, s, static_cast<const T *>(b.q), static_cast<const T *>(b.cache),
                       static_cast<T *>(b.o), b.ldo, rw, b.bias, d.bias_len, d.heads, d.kv_heads, d.dim, d.vdim, d.ring, d.window, d.scale, d.out_scale);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    };
    if (d.vdim <= 64) return go(attn_rows_kernel<T, 2>);
    if (d.vdim <= 128) return go(attn_rows_kernel<T, 4>);
    if (d.vdim <= 256) return go(attn_rows_kernel<T, 8>);
    return go(attn_rows_kernel<T, 32>);
}

int decode(smc_ctx *ctx, const smc_attn_dims &d, const smc_attn_bufs &b, const smc_rows &rw, cudaStream_t s)
{
    const int smem = decode_smem(d.dim, d.vdim), per_sm = smem <= 110 * 1024 ? 2 : 1;
    const int groups = d.kv_heads * ((d.heads / d.kv_heads + 15) / 16);
    // as many CTAs per row as keep the device full, up to the cluster limit and to one tile per warp
    const int most = ((d.window > 0 ? d.window : d.ring) + DKT * DWP - 1) / (DKT * DWP);
    int cl = DCL;
    while (cl > 1 && ((long long)rw.n * groups * cl > (long long)per_sm * ctx->sm_count || cl / 2 >= most)) cl /= 2;
    const bool half = d.heads / d.kv_heads <= 8, reg = d.dim <= 128;
    return by_value_tiles(d.vdim, [&](auto vt) {
        constexpr int VT = decltype(vt)::value;
        auto kernel = half ? (reg ? attn_decode_kernel<VT, true, 8> : attn_decode_kernel<VT, true, 0>)
                           : (reg ? attn_decode_kernel<VT, false, 8> : attn_decode_kernel<VT, false, 0>);
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        smc_launch_dep_cluster(ctx->use_pdl, cl, kernel, dim3(cl, groups, rw.n), dim3(DWP * 32), smem, s, static_cast<const bf16 *>(b.in), b.ld, b.col,
                               static_cast<bf16 *>(b.cache), static_cast<bf16 *>(b.o), b.ldo, rw, b.q_norm, b.k_norm, b.bias, d.bias_len, d.heads,
                               d.kv_heads, d.dim, d.vdim, d.ring, d.window, d.scale, d.out_scale, d.eps);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    });
}

int prefill(smc_ctx *ctx, const smc_attn_dims &d, const smc_attn_bufs &b, const smc_rows &rw, int pos0, cudaStream_t s)
{
    int rc = post<bf16>(ctx, d, b, rw, s);
    if (rc) return rc;
    const int smem = prefill_smem(d.dim, d.vdim);
    return by_value_tiles(d.vdim, [&](auto vt) {
        auto kernel = attn_prefill_kernel<decltype(vt)::value>;
        SMC_CUDA(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        smc_launch_dep(ctx->use_pdl, kernel, dim3(d.heads, (rw.n + PQ - 1) / PQ), dim3(128), smem, s, static_cast<const bf16 *>(b.q),
                       static_cast<const bf16 *>(b.cache), static_cast<bf16 *>(b.o), b.ldo, b.bias, d.bias_len, rw.n, rw.seq0, pos0, d.heads, d.kv_heads,
                       d.dim, d.vdim, d.ring, d.window, d.scale, d.out_scale);
        SMC_LAUNCH_CHECK(ctx);
        return (int)SMC_OK;
    });
}

}  // namespace

int smc_attn_check(smc_ctx *ctx, const smc_attn_dims &d)
{
    if (d.dim > 2048 || d.vdim > 1024) return smc_fail(ctx, SMC_E_UNSUPPORTED, "attention heads of %d / %d (up to 2048 / 1024 are built)", d.dim, d.vdim);
    return SMC_OK;
}

int smc_attn_mix(smc_ctx *ctx, const smc_attn_dims &d, const smc_attn_bufs &b, const smc_rows &rw, int is_bf16, int pos0, cudaStream_t s)
{
    if (!is_bf16) return rows<float>(ctx, d, b, rw, s);
    constexpr int MOST = 220 * 1024;
    const bool one = rw.seq0 < 0 || rw.n == 1;
    const bool fours = b.ld % 4 == 0 && b.col % 4 == 0 && whole(b.in) && whole(b.q_norm) && whole(b.k_norm);
    if (pieces_fit(d, b) && fours && one && decode_smem(d.dim, d.vdim) <= MOST) return decode(ctx, d, b, rw, s);
    if (pieces_fit(d, b) && !one && prefill_smem(d.dim, d.vdim) <= MOST) return prefill(ctx, d, b, rw, pos0, s);
    return rows<bf16>(ctx, d, b, rw, s);
}

int smc_attn_expand_bias(smc_ctx *ctx, const float *table, int heads, int buckets, double bias_max, int len, float *out, cudaStream_t s)
{
    std::vector<int> bucket(len);
    const int half = buckets / 2;
    for (int n = 0; n < len; ++n) {
        bucket[n] = n;
        if (n >= half) {
            const double far = half + floor(log((double)n / half) / log(bias_max / half) * (buckets - half));
            bucket[n] = far < buckets - 1 ? (int)far : buckets - 1;
        }
    }
    int *d_bucket = nullptr;
    SMC_CUDA(ctx, cudaMalloc(&d_bucket, (size_t)len * sizeof(int)));
    cudaError_t e = cudaMemcpy(d_bucket, bucket.data(), (size_t)len * sizeof(int), cudaMemcpyHostToDevice);
    if (e == cudaSuccess) {
        expand_bias_kernel<<<(unsigned)(((long long)heads * len + 255) / 256), 256, 0, s>>>(table, d_bucket, heads, len, out);
        e = cudaGetLastError();
    }
    if (e == cudaSuccess) e = cudaStreamSynchronize(s);
    cudaFree(d_bucket);
    return e == cudaSuccess ? (int)SMC_OK : smc_fail(ctx, SMC_E_CUDA, "expand_bias: %s", cudaGetErrorString(e));
}
