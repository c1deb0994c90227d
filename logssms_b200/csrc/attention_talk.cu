// Attention whose heads mix their softmax weights, on the tensor cores (bfloat16): the sums of every query head's weights over
// the values of ALL key/value heads.
//
//   Query head g (of Hq) scores the keys of key/value head g / (Hq / Hkv); position i sees the tokens j <= i with i - j < window or
//   j < keep.  With w_g(i, j) its softmax weights, the kernels here leave, per token and head,
//       U_g(i) = sum_j w_g(i, j) [v_0(j) | v_1(j) | ...]        (a row of Hkv * vdim columns)
//   unnormalized, with the maximum and the sum of the weights, per key range; `talk_merge` (attention_pooled.cu) joins the ranges and
//   the sink, divides and mixes: head h of key/value head c is sum_g M[h, g] U_g's columns of c.
//
//   talk_tile : prompt portions: a CTA per (run of up to 64 neighbouring tokens of a request, query head, key range)
//   talk_step : decoded tokens and short portions: a CTA per (token, 16 query heads, key range); a staged key/value row serves all
//               of them
//
// Scores, maxima, weights and sums are float32.  A weight p enters the product with the values as the two bfloat16 terms hi =
// bf16(p), lo = bf16(p - hi) (two `mma.sync` into one accumulator), so it is applied to 16 bits and more, not rounded to 8.
#include "lb200/common.cuh"
using namespace lb200;

typedef __nv_bfloat16 bf16;
constexpr int kOff = 8;                  // floats in front of the value columns of a partial result (kTalkOff of attention_pooled.cu)
constexpr float kLog2e = 1.4426950408889634f, kLn2 = 0.6931471805599453f;

__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool live) {       // 16 bytes, or zeros
    const int bytes = live ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void copies_done() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// two weights as two bfloat16 terms each
__device__ __forceinline__ void two_terms(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// the cache row of entry number kk: the `lead` kept tokens first, then the tokens from `first` on; -1: no page
__device__ __forceinline__ long cache_row(int kk, int lead, int first, const int* __restrict__ pages, int page_size) {
    const int e = kk < lead ? kk : first + (kk - lead);
    const int page = pages[e / page_size];
    return page < 0 ? -1 : (long)page * page_size + e % page_size;
}

__device__ __forceinline__ float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

// ------------------------------------------------------------------------------------------------ prompt portions
// 16 warps: rw = warp % 4 owns 16 of the run's 64 query rows, cw = warp / 4 a quarter of the CTA's value columns (NT tiles of 8)
// and a quarter of a chunk's 64 keys.  Per chunk a warp scores its 16 keys, the four warps of a row tile agree on the rows'
// maxima through shared memory, each leaves its weights (two bfloat16 planes) there, and then multiplies all 64 keys' weights
// with its columns.  The chunks alternate between two buffers (`cp.async`).  Scores are kept in the base-2 domain.
constexpr int kRun = 64, kKeys = 64, kTileThreads = 512;

template <int NT>
__global__ void __launch_bounds__(kTileThreads, NT <= 4 ? 2 : 1) talk_tile_kernel(
        const bf16* __restrict__ q, const bf16* __restrict__ k_cache, const bf16* __restrict__ v_cache, const int* __restrict__ block_table,
        int table_width, const int* __restrict__ cu, const int* __restrict__ start_pos, const int* __restrict__ tiles, int num_tiles,
        float* __restrict__ partial, int Hq, int Hkv, int dim, int width, int page_size, float scale2, int window, int keep, int splits) {
    extern __shared__ __align__(16) unsigned char smem[];
    // the runs that see most keys come last in the list: they start first
    const int tile = num_tiles - 1 - (int)blockIdx.y, split = blockIdx.z;
    const int head = blockIdx.x % Hq, v_col = (blockIdx.x / Hq) * (NT * 32);
    const int b = tiles[2 * tile];
    if (b < 0) return;
    const int t0 = tiles[2 * tile + 1];
    const int cols = min(NT * 32, width - v_col);
    const int g = head / (Hq / Hkv);
    const int n_q = min(kRun, cu[b + 1] - cu[b] - t0);
    const int row0 = cu[b] + t0, pos0 = start_pos[b] + t0, i_last = pos0 + n_q - 1;
    const int first = max(0, pos0 - window + 1);                    // the oldest token any query of the run sees in its window
    const int lead = min(keep, first);                              // kept tokens behind that: every query sees them
    const int keys = lead + (i_last - first + 1);
    const int k_stride = dim + 8, v_stride = NT * 32 + 8, p_stride = kKeys + 8;      // elements; the pads stagger the banks
    bf16* Qs = reinterpret_cast<bf16*>(smem);                       // [64][k_stride]
    bf16* Ks = Qs + kRun * k_stride;                                // [2][64][k_stride]
    bf16* Vs = Ks + 2 * kKeys * k_stride;                           // [2][64][v_stride]
    bf16* Ps = Vs + 2 * kKeys * v_stride;                           // [2 terms][64][p_stride]
    float* maxima = reinterpret_cast<float*>(Ps + 2 * kRun * p_stride);      // [4 cw][64]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rw = warp & 3, cw = warp >> 2, gq = lane >> 2, tq = lane & 3;
    const int dsteps = dim / 16;
    const int* pages = block_table + (size_t)b * table_width;

    // a chunk's rows: 8 threads per key row, first the keys' pieces, then the values'
    const int pk = dim / 8, pv = cols / 8;
    auto prefetch = [&](int k0, int buf) {
        const int r = threadIdx.x >> 3, part = threadIdx.x & 7, kk = k0 + r;
        const long row = kk < keys ? cache_row(kk, lead, first, pages, page_size) : -1;
        const bool live = row >= 0;
        const bf16* ks = k_cache + (live ? ((size_t)row * Hkv + g) * dim : 0);
        const bf16* vs = v_cache + (live ? (size_t)row * width + v_col : 0);
        const uint32_t kd = smem_addr(Ks + ((size_t)buf * kKeys + r) * k_stride), vd = smem_addr(Vs + ((size_t)buf * kKeys + r) * v_stride);
        for (int p = part; p < pk; p += 8) copy16(kd + p * 16, live ? ks + p * 8 : ks, live);
        for (int p = part; p < pv; p += 8) copy16(vd + p * 16, live ? vs + p * 8 : vs, live);
        copies_done();
    };
    const int chunks_all = (keys + kKeys - 1) / kKeys, chunks_per = (chunks_all + splits - 1) / splits;
    const int k_first = min(keys, split * chunks_per * kKeys), k_last = min(keys, k_first + chunks_per * kKeys);
    if (k_first < k_last) prefetch(k_first, 0);
    for (int i = threadIdx.x; i < kRun * pk; i += kTileThreads) {
        const int r = i / pk, p = i % pk;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < n_q) v = *reinterpret_cast<const uint4*>(q + ((size_t)(row0 + r) * Hq + head) * dim + p * 8);
        *reinterpret_cast<uint4*>(Qs + r * k_stride + p * 8) = v;
    }
    // fragment addresses: ldmatrix takes lane l's row of matrix l / 8
    const int mi = lane >> 3, mr = lane & 7;
    const uint32_t q_addr = smem_addr(Qs + (rw * 16 + (mi & 1) * 8 + mr) * k_stride + (mi >> 1) * 8);
    const uint32_t k_addr = smem_addr(Ks + (cw * 16 + (mi >> 1) * 8 + mr) * k_stride + (mi & 1) * 8);
    const uint32_t v_addr = smem_addr(Vs + ((mi & 1) * 8 + mr) * v_stride + cw * NT * 8 + (mi >> 1) * 8);
    const uint32_t p_addr = smem_addr(Ps + (rw * 16 + (mi & 1) * 8 + mr) * p_stride + (mi >> 1) * 8);
    const int iw0 = pos0 + rw * 16, iw1 = min(iw0 + 15, i_last);    // this row tile's positions
    const int i_lo = iw0 + gq, i_hi = i_lo + 8;
    const int live_cols = cols - cw * NT * 8;                       // value columns of this warp that exist
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int k0 = k_first, it = 0; k0 < k_last; k0 += kKeys, ++it) {
        copies_wait();
        __syncthreads();                             // this chunk has landed; the chunk before is consumed by every warp
        if (k0 + kKeys < k_last) prefetch(k0 + kKeys, (it + 1) & 1);
        // the chunk's tokens: is any of them visible to a row of this tile, are all of them visible to all rows?
        const int c_last = min(k0 + kKeys, keys) - 1;
        const int ja = first + max(k0 - lead, 0), jb = first + c_last - lead;       // window tokens of the chunk (none: jb < first)
        const bool any = k0 < lead || ((jb > iw0 - window || ja < keep) && ja <= iw1);
        if (!any || iw0 > i_last) continue;          // (the four warps of a row tile agree)
        const bool all = c_last - k0 == kKeys - 1 && (c_last < lead || (jb <= iw0 && ja > iw1 - window));
        const uint32_t kb = k_addr + (uint32_t)((it & 1) * kKeys * k_stride * 2);
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
        for (int ks = 0; ks < dsteps; ++ks) {
            uint32_t a[4], kf[4];
            ldsm(a, q_addr + ks * 32);
            ldsm(kf, kb + ks * 32);
            mma(s[0], a, kf[0], kf[1]);
            mma(s[1], a, kf[2], kf[3]);
        }
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                float v = s[n][x] * scale2;
                if (!all) {
                    const int kk = k0 + cw * 16 + n * 8 + 2 * tq + (x & 1), i = x >= 2 ? i_hi : i_lo;
                    const int j = first + kk - lead;
                    const bool seen = kk < keys && i <= i_last && (kk < lead || (j <= i && (j > i - window || j < keep)));
                    v = seen ? v : -INFINITY;
                }
                s[n][x] = v;
                if (x >= 2) mx_hi = fmaxf(mx_hi, v); else mx_lo = fmaxf(mx_lo, v);
            }
        }
        mx_lo = quad_max(mx_lo); mx_hi = quad_max(mx_hi);
        if (tq == 0) { maxima[cw * kRun + rw * 16 + gq] = mx_lo; maxima[cw * kRun + rw * 16 + gq + 8] = mx_hi; }
        asm volatile("bar.sync %0, 128;" ::"r"(1 + rw) : "memory");
        float mn_lo = m_lo, mn_hi = m_hi;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            mn_lo = fmaxf(mn_lo, maxima[w * kRun + rw * 16 + gq]);
            mn_hi = fmaxf(mn_hi, maxima[w * kRun + rw * 16 + gq + 8]);
        }
        const float base_lo = mn_lo == -INFINITY ? 0.f : mn_lo, base_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
        const float c_lo = exp2f(m_lo - base_lo), c_hi = exp2f(m_hi - base_hi);      // (nothing seen before: exp2(-inf) = 0)
        const bool moved = m_lo != mn_lo || m_hi != mn_hi;
        m_lo = mn_lo; m_hi = mn_hi;
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const float p0 = exp2f(s[n][0] - base_lo), p1 = exp2f(s[n][1] - base_lo), p2 = exp2f(s[n][2] - base_hi), p3 = exp2f(s[n][3] - base_hi);
            sum_lo += p0 + p1; sum_hi += p2 + p3;
            uint32_t h0, l0, h1, l1;
            two_terms(p0, p1, h0, l0);
            two_terms(p2, p3, h1, l1);
            bf16* at = Ps + (rw * 16 + gq) * p_stride + cw * 16 + n * 8 + 2 * tq;
            *reinterpret_cast<uint32_t*>(at) = h0;
            *reinterpret_cast<uint32_t*>(at + 8 * p_stride) = h1;
            *reinterpret_cast<uint32_t*>(at + kRun * p_stride) = l0;
            *reinterpret_cast<uint32_t*>(at + (kRun + 8) * p_stride) = l1;
        }
        l_lo = l_lo * c_lo + sum_lo;                 // (this thread's keys only: the lanes' and warps' sums meet at the end)
        l_hi = l_hi * c_hi + sum_hi;
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int n = 0; n < NT; ++n) { o[n][0] *= c_lo; o[n][1] *= c_lo; o[n][2] *= c_hi; o[n][3] *= c_hi; }
        }
        asm volatile("bar.sync %0, 128;" ::"r"(1 + rw) : "memory");
        const uint32_t vb = v_addr + (uint32_t)((it & 1) * kKeys * v_stride * 2);
#pragma unroll
        for (int ks = 0; ks < kKeys / 16; ++ks) {
            uint32_t ph[4], pl[4];
            ldsm(ph, p_addr + ks * 32);
            ldsm(pl, p_addr + kRun * p_stride * 2 + ks * 32);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                if (n * 8 >= live_cols) continue;
                uint32_t vf[4];
                ldsm_trans(vf, vb + ks * 16 * v_stride * 2 + n * 16);
                mma(o[n], ph, vf[0], vf[1]);
                mma(o[n + 1], ph, vf[2], vf[3]);
                mma(o[n], pl, vf[0], vf[1]);
                mma(o[n + 1], pl, vf[2], vf[3]);
            }
        }
    }
    // the four key quarters' sums meet (a warp without work leaves its zeros)
    __syncthreads();
    l_lo = quad_sum(l_lo); l_hi = quad_sum(l_hi);
    if (tq == 0) { maxima[cw * kRun + rw * 16 + gq] = l_lo; maxima[cw * kRun + rw * 16 + gq + 8] = l_hi; }
    __syncthreads();
    const int r_lo = rw * 16 + gq, r_hi = r_lo + 8, stride = width + kOff;
    float* p_lo = partial + (((size_t)(row0 + r_lo) * Hq + head) * splits + split) * stride;
    float* p_hi = partial + (((size_t)(row0 + r_hi) * Hq + head) * splits + split) * stride;
    if (cw == 0 && tq == 0 && v_col == 0) {
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) { sum_lo += maxima[w * kRun + r_lo]; sum_hi += maxima[w * kRun + r_hi]; }
        if (r_lo < n_q) { p_lo[0] = m_lo * kLn2; p_lo[1] = sum_lo; }
        if (r_hi < n_q) { p_hi[0] = m_hi * kLn2; p_hi[1] = sum_hi; }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        if (n * 8 >= live_cols) continue;
        const int c = kOff + v_col + (cw * NT + n) * 8 + 2 * tq;
        if (r_lo < n_q) *reinterpret_cast<float2*>(p_lo + c) = make_float2(o[n][0], o[n][1]);
        if (r_hi < n_q) *reinterpret_cast<float2*>(p_hi + c) = make_float2(o[n][2], o[n][3]);
    }
}

static size_t tile_smem(int nt, int dim) {
    return ((size_t)3 * kRun * (dim + 8) + (size_t)2 * kKeys * (nt * 32 + 8) + (size_t)2 * kRun * (kKeys + 8)) * sizeof(bf16)
         + (size_t)4 * kRun * sizeof(float);
}

extern "C" int lb_talk_tile_q() { return kRun; }

// q: [tokens, Hq, dim]; caches [slots, Hkv, dim], [slots, Hkv, vdim]; tiles: int32 [num_tiles, 2] (request, first token of the run
// within its portion; request -1: no work); partial: float32 [tokens, Hq, splits, Hkv * vdim + 8], the runs' rows are written.
// dim: a multiple of 16 up to 128, vdim: a multiple of 8
extern "C" int lb_talk_tile(const void* q, const void* k_cache, const void* v_cache, const int* block_table, int table_width, const int* cu,
                            const int* start_pos, const int* tiles, int num_tiles, float* partial, int Hq, int Hkv, int dim, int vdim,
                            int page_size, float scale, int window, int keep, int splits, void* stream) {
    if (num_tiles <= 0) return kOk;
    if (Hq <= 0 || Hkv <= 0 || Hq % Hkv || dim <= 0 || dim % 16 || vdim <= 0 || vdim % 8 || page_size <= 0 || window <= 0 || keep < 0
        || splits <= 0 || splits > 64)
        return kBadSize;
    const int width = Hkv * vdim;
    const long chunks = (width + 511) / 512;
    if (dim > 128 || num_tiles > 65535 || Hq * chunks > (1L << 30)) return kTooLarge;
    const float scale2 = scale * kLog2e;
#define LB_TILE(NT) { const size_t smem = tile_smem(NT, dim); static size_t have = 0; ensure_dynamic_smem(talk_tile_kernel<NT>, smem, have); \
        talk_tile_kernel<NT><<<dim3((unsigned)(Hq * ((width + NT * 32 - 1) / (NT * 32))), num_tiles, splits), kTileThreads, smem, (cudaStream_t)stream>>>( \
            (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, block_table, table_width, cu, start_pos, tiles, num_tiles, partial, Hq, Hkv, \
            dim, width, page_size, scale2, window, keep, splits); }
    if (width <= 128) LB_TILE(4) else if (width <= 256) LB_TILE(8) else LB_TILE(16)
#undef LB_TILE
    return launch_status();
}

// ------------------------------------------------------------------------------------------------ decoded tokens
// 8 warps; the 16 rows of a tile are 16 query heads of the token (a last tile may have fewer).  Per chunk of KC keys: warp w scores
// the 8 keys w % (KC / 8) against every (8 / (KC / 8))-th key/value head, all 16 rows at once, and keeps the rows of the heads that
// belong to it; the scores meet in shared memory; every warp then makes all weights from them and multiplies with its own NT * 8
// value columns.  The chunks alternate between two buffers (`cp.async`).
constexpr int kStepThreads = 256;

// key/value heads that 16 neighbouring query heads can belong to
__host__ __device__ __forceinline__ int most_kv_heads(int per, int Hkv) {
    const int n = (16 + per - 1) / per + 1;
    return n < Hkv ? n : Hkv;
}

template <int NT, int KC>
__global__ void __launch_bounds__(kStepThreads) talk_step_kernel(
        const bf16* __restrict__ q, const bf16* __restrict__ k_cache, const bf16* __restrict__ v_cache, const int* __restrict__ block_table,
        int table_width, const int* __restrict__ token_req, const int* __restrict__ positions, const int* __restrict__ token_list,
        float* __restrict__ partial, int Hq, int Hkv, int dim, int width, int page_size, float scale2, int window, int keep, int splits) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int kTiles = KC / 8, kParts = 8 / kTiles;             // key tiles of a chunk; warps that share one
    const int slot = blockIdx.x, split = blockIdx.z;
    const int t = token_list != nullptr ? token_list[slot] : slot;
    if (t < 0) return;
    const int head_tiles = (Hq + 15) / 16;
    const int h0 = (blockIdx.y % head_tiles) * 16, nh = min(16, Hq - h0), v_col = (blockIdx.y / head_tiles) * (NT * 64);
    const int per = Hq / Hkv, g0 = h0 / per, ng = (h0 + nh - 1) / per - g0 + 1;       // key/value heads of the tile
    const int cols = min(NT * 64, width - v_col);
    const int pos = positions[t], first = max(0, pos - window + 1), lead = min(keep, first), keys = lead + (pos - first + 1);
    const int* pages = block_table + (size_t)token_req[t] * table_width;
    const int q_stride = dim + 8, k_stride = ng * dim + 8, v_stride = NT * 64 + 8;
    const int k_room = most_kv_heads(per, Hkv) * dim + 8;           // (the stride is at most this: the buffers are laid out for it)
    constexpr int s_stride = KC + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem);                       // [16][q_stride]
    bf16* Ks = Qs + 16 * q_stride;                                  // [2][KC][k_stride]
    bf16* Vs = Ks + 2 * KC * k_room;                                // [2][KC][v_stride]
    float* Ss = reinterpret_cast<float*>(Vs + 2 * KC * v_stride);   // [16][s_stride]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gq = lane >> 2, tq = lane & 3;
    const int dsteps = dim / 16, pk = ng * dim / 8, pv = cols / 8;
    constexpr int kLanes = kStepThreads / KC;                       // threads per key row
    auto prefetch = [&](int k0, int k_end, int buf) {
        const int r = threadIdx.x / kLanes, part = threadIdx.x % kLanes, kk = k0 + r;
        const long row = kk < k_end ? cache_row(kk, lead, first, pages, page_size) : -1;
        const bool live = row >= 0;
        const bf16* ks = k_cache + (live ? ((size_t)row * Hkv + g0) * dim : 0);
        const bf16* vs = v_cache + (live ? (size_t)row * width + v_col : 0);
        const uint32_t kd = smem_addr(Ks + ((size_t)buf * KC + r) * k_stride), vd = smem_addr(Vs + ((size_t)buf * KC + r) * v_stride);
        for (int p = part; p < pk; p += kLanes) copy16(kd + p * 16, live ? ks + p * 8 : ks, live);
        for (int p = part; p < pv; p += kLanes) copy16(vd + p * 16, live ? vs + p * 8 : vs, live);
        copies_done();
    };
    const int chunks_all = (keys + KC - 1) / KC, chunks_per = (chunks_all + splits - 1) / splits;
    const int k_first = min(keys, split * chunks_per * KC), k_last = min(keys, k_first + chunks_per * KC);
    if (k_first < k_last) prefetch(k_first, k_last, 0);
    const int pq = dim / 8;
    for (int i = threadIdx.x; i < 16 * pq; i += kStepThreads) {
        const int r = i / pq, p = i % pq;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < nh) v = *reinterpret_cast<const uint4*>(q + ((size_t)t * Hq + h0 + r) * dim + p * 8);
        *reinterpret_cast<uint4*>(Qs + r * q_stride + p * 8) = v;
    }
    const int mi = lane >> 3, mr = lane & 7;
    const int kt = warp % kTiles, part0 = warp / kTiles;
    const uint32_t q_addr = smem_addr(Qs + ((mi & 1) * 8 + mr) * q_stride + (mi >> 1) * 8);
    // key fragments of two k-steps at a time: matrices (dims 0-7, 8-15) of the step, then of the next one
    const uint32_t k_addr = smem_addr(Ks + (kt * 8 + mr) * k_stride + (mi >> 1) * 16 + (mi & 1) * 8);
    const uint32_t v_addr = smem_addr(Vs + ((mi & 1) * 8 + mr) * v_stride + warp * NT * 8 + (mi >> 1) * 8);
    const int live_cols = cols - warp * NT * 8;
    const int g_lo = (h0 + min(gq, nh - 1)) / per - g0, g_hi = (h0 + min(gq + 8, nh - 1)) / per - g0;      // the rows' key/value heads
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int k0 = k_first, it = 0; k0 < k_last; k0 += KC, ++it) {
        copies_wait();
        __syncthreads();                             // this chunk has landed; the chunk before and its scores are consumed
        if (k0 + KC < k_last) prefetch(k0 + KC, k_last, (it + 1) & 1);
        const uint32_t kb = k_addr + (uint32_t)((it & 1) * KC * k_stride * 2);
        for (int g = part0; g < ng; g += kParts) {
            float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
            int ks = 0;
#pragma unroll 4
            for (; ks + 2 <= dsteps; ks += 2) {
                uint32_t a[4], a2[4], kf[4];
                ldsm(a, q_addr + ks * 32);
                ldsm(a2, q_addr + ks * 32 + 32);
                ldsm(kf, kb + (g * dim + ks * 16) * 2);
                mma(s, a, kf[0], kf[1]);
                mma(s2, a2, kf[2], kf[3]);
            }
            if (ks < dsteps) {                       // (the second pair of matrices may lie behind the head: read, not used)
                uint32_t a[4], kf[4];
                ldsm(a, q_addr + ks * 32);
                ldsm(kf, kb + (g * dim + ks * 16) * 2);
                mma(s, a, kf[0], kf[1]);
            }
            const int kk = k0 + kt * 8 + 2 * tq;
            const float e0 = kk < k_last ? scale2 : -INFINITY, e1 = kk + 1 < k_last ? scale2 : -INFINITY;
            float* at = Ss + gq * s_stride + kt * 8 + 2 * tq;
            if (g_lo == g) *reinterpret_cast<float2*>(at) = make_float2(e0 == -INFINITY ? e0 : (s[0] + s2[0]) * e0, e1 == -INFINITY ? e1 : (s[1] + s2[1]) * e1);
            if (g_hi == g) *reinterpret_cast<float2*>(at + 8 * s_stride) = make_float2(e0 == -INFINITY ? e0 : (s[2] + s2[2]) * e0, e1 == -INFINITY ? e1 : (s[3] + s2[3]) * e1);
        }
        __syncthreads();
        // every warp: the weights of all rows in the layout of the next product's first operand
        float p[KC / 8][4];
        float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
        for (int n = 0; n < KC / 8; ++n) {
            const float2 lo = *reinterpret_cast<const float2*>(Ss + gq * s_stride + n * 8 + 2 * tq);
            const float2 hi = *reinterpret_cast<const float2*>(Ss + (gq + 8) * s_stride + n * 8 + 2 * tq);
            p[n][0] = lo.x; p[n][1] = lo.y; p[n][2] = hi.x; p[n][3] = hi.y;
            mx_lo = fmaxf(mx_lo, fmaxf(lo.x, lo.y)); mx_hi = fmaxf(mx_hi, fmaxf(hi.x, hi.y));
        }
        mx_lo = quad_max(mx_lo); mx_hi = quad_max(mx_hi);            // (a chunk has a key: finite)
        const float c_lo = exp2f(m_lo - mx_lo), c_hi = exp2f(m_hi - mx_hi);
        m_lo = mx_lo; m_hi = mx_hi;
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int n = 0; n < KC / 8; ++n) {
            p[n][0] = exp2f(p[n][0] - mx_lo); p[n][1] = exp2f(p[n][1] - mx_lo);
            p[n][2] = exp2f(p[n][2] - mx_hi); p[n][3] = exp2f(p[n][3] - mx_hi);
            sum_lo += p[n][0] + p[n][1]; sum_hi += p[n][2] + p[n][3];
        }
        l_lo = l_lo * c_lo + sum_lo; l_hi = l_hi * c_hi + sum_hi;
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[n][0] *= c_lo; o[n][1] *= c_lo; o[n][2] *= c_hi; o[n][3] *= c_hi; }
        const uint32_t vb = v_addr + (uint32_t)((it & 1) * KC * v_stride * 2);
#pragma unroll
        for (int ks = 0; ks < KC / 16; ++ks) {
            uint32_t ph[4], pl[4];
            two_terms(p[2 * ks][0], p[2 * ks][1], ph[0], pl[0]);
            two_terms(p[2 * ks][2], p[2 * ks][3], ph[1], pl[1]);
            two_terms(p[2 * ks + 1][0], p[2 * ks + 1][1], ph[2], pl[2]);
            two_terms(p[2 * ks + 1][2], p[2 * ks + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                if (n * 8 >= live_cols) continue;
                uint32_t vf[4];
                ldsm_trans(vf, vb + ks * 16 * v_stride * 2 + n * 16);
                mma(o[n], ph, vf[0], vf[1]);
                mma(o[n + 1], ph, vf[2], vf[3]);
                mma(o[n], pl, vf[0], vf[1]);
                mma(o[n + 1], pl, vf[2], vf[3]);
            }
        }
    }
    l_lo = quad_sum(l_lo); l_hi = quad_sum(l_hi);
    const int stride = width + kOff;
    float* p_lo = partial + (((size_t)slot * Hq + h0 + gq) * splits + split) * stride;
    float* p_hi = partial + (((size_t)slot * Hq + h0 + gq + 8) * splits + split) * stride;
    if (warp == 0 && tq == 0 && v_col == 0) {
        if (gq < nh) { p_lo[0] = m_lo * kLn2; p_lo[1] = l_lo; }
        if (gq + 8 < nh) { p_hi[0] = m_hi * kLn2; p_hi[1] = l_hi; }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        if (n * 8 >= live_cols) continue;
        const int c = kOff + v_col + (warp * NT + n) * 8 + 2 * tq;
        if (gq < nh) *reinterpret_cast<float2*>(p_lo + c) = make_float2(o[n][0], o[n][1]);
        if (gq + 8 < nh) *reinterpret_cast<float2*>(p_hi + c) = make_float2(o[n][2], o[n][3]);
    }
}

static size_t step_smem(int nt, int kc, int per, int Hkv, int dim) {
    const int k_room = most_kv_heads(per, Hkv) * dim + 8;
    return ((size_t)16 * (dim + 8) + (size_t)2 * kc * k_room + (size_t)2 * kc * (nt * 64 + 8)) * sizeof(bf16) + (size_t)16 * (kc + 8) * sizeof(float);
}
static int step_columns(int width) { return width <= 128 ? 2 : (width <= 256 ? 4 : 8); }       // value tiles of 8 columns per warp
constexpr size_t kStepMaxSmem = 200 * 1024;

// does `lb_talk_step` take these sizes?
extern "C" int lb_talk_step_ok(int Hq, int Hkv, int dim, int vdim) {
    if (Hq <= 0 || Hkv <= 0 || Hq % Hkv || dim <= 0 || dim % 16 || dim > 256 || vdim <= 0 || vdim % 8) return 0;
    return step_smem(step_columns(Hkv * vdim), 16, Hq / Hkv, Hkv, dim) <= kStepMaxSmem;
}

// As `lb_talk_tile` for single tokens (all of the step's, or those of `token_list`); partial: float32 [num_tokens, Hq, splits,
// Hkv * vdim + 8], row by row of the list.  dim: a multiple of 16 up to 256, vdim: a multiple of 8 (see `lb_talk_step_ok`)
extern "C" int lb_talk_step(const void* q, const void* k_cache, const void* v_cache, const int* block_table, int table_width,
                            const int* token_req, const int* positions, const int* token_list, int num_tokens, float* partial, int Hq, int Hkv,
                            int dim, int vdim, int page_size, float scale, int window, int keep, int splits, void* stream) {
    if (num_tokens <= 0) return kOk;
    if (!lb_talk_step_ok(Hq, Hkv, dim, vdim) || page_size <= 0 || window <= 0 || keep < 0 || splits <= 0 || splits > 65535) return kBadSize;
    const int width = Hkv * vdim, nt = step_columns(width), per = Hq / Hkv;
    const float scale2 = scale * kLog2e;
    const long rows = (long)((Hq + 15) / 16) * ((width + nt * 64 - 1) / (nt * 64));
    if (rows > 65535) return kTooLarge;
    const bool wide = step_smem(nt, 32, per, Hkv, dim) <= kStepMaxSmem;             // chunks of 32 keys, or of 16 where those are too large
#define LB_STEP(NT, KC) { const size_t smem = step_smem(NT, KC, per, Hkv, dim); static size_t have = 0; ensure_dynamic_smem(talk_step_kernel<NT, KC>, smem, have); \
        talk_step_kernel<NT, KC><<<dim3(num_tokens, (unsigned)rows, splits), kStepThreads, smem, (cudaStream_t)stream>>>( \
            (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, block_table, table_width, token_req, positions, token_list, partial, Hq, Hkv, \
            dim, width, page_size, scale2, window, keep, splits); }
    if (wide) { if (nt == 2) LB_STEP(2, 32) else if (nt == 4) LB_STEP(4, 32) else LB_STEP(8, 32) }
    else { if (nt == 2) LB_STEP(2, 16) else if (nt == 4) LB_STEP(4, 16) else LB_STEP(8, 16) }
#undef LB_STEP
    return launch_status();
}
