// Routed feed-forward: the router, the experts' activation, identity experts, and the tanh GELU of dense layers.
//
//  moe_route        : 32-bit router per token: logits = W_r h, s = softmax over all n outputs (real and identity
//                     experts alike), or with `sigmoid_scores` s = sigmoid of each logit; the choice looks at
//                     s + correction (if there is one), restricted to the `keep` groups (of
//                     n / groups neighbours) whose best member scores highest; the `top` best are chosen; their
//                     weights are s * scale (no correction, no renormalisation).  With `sigmoid_scores` = 2 the
//                     logits themselves are ranked and the chosen ones' weights are the softmax over the chosen
//                     logits only (times scale).  `bias` (may be null) is added to the logits.  With `pair_groups` a
//                     group's score is the sum of its two largest members instead of its largest; with `normalize` the
//                     chosen weights are divided by their sum + 1e-20; `gates` further rows of W_r behind the n outputs
//                     are no experts: the dense weights' last `gates` columns are the sigmoids of their logits.  Writes the dense weights [T, n + gates]
//                     (0 where not chosen), the chosen indices and weights [T, top], and per token the summed
//                     weight of the chosen identity experts (the last n - experts outputs).
//  moe_activation   : y[t, e, i] = w[t, e] * g~ * sigmoid(act_alpha * g~) * (u~ + 1),  g~ = min(g, limit),
//                     u~ = clamp(u, -limit, limit), from the packed [gate | up] products of all experts.  The expert's
//                     weight is applied here, so ONE product with the stacked down matrices sums the experts.
//                     Mode `kSiluInput`: y = silu(w g) * (w u), the expert silu(gate) * up on an input that was
//                     multiplied by the weight (gate and up are linear in it).  Without weights (`dense` null, one
//                     expert) it is the activation of a dense gated layer.  Modes `kSiluOutput` and `kGeluOutput`:
//                     y = w * silu(g) * u and y = w * gelu_tanh(g) * u.  Input and output rows may be column views
//                     of wider matrices (row strides in elements).  `tail_ff` > 0: behind the experts' columns lies one
//                     more expert of that size (input gate | up, output), whose weight is dense column `tail_gate`, or 1.
//  moe_add_identity : out += id_weight[t] * h
//  gelu_tanh        : 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
//  xielu            : a z^2 + z/2 for z > 0, b (e^z - 1 - z) + z/2 for z <= 0, with a and b read from memory
#include "lb200/common.cuh"
using namespace lb200;

constexpr int kRouteMax = 256;        // router outputs
// warps of a CTA, which share the router outputs: one token per CTA (few tokens) takes many, several tokens fewer with more
// registers each, so that more loads are in flight
constexpr int route_warps(int tok) { return tok == 1 ? 16 : 8; }

// the index of the largest v[i] among those with ok[i] (ties: the lower index), -1 if there is none; by one warp, all lanes get it
__device__ __forceinline__ int warp_best(const float* v, const unsigned char* ok, int n) {
    unsigned key = 0, at = 0xffffffffu;                    // floats as unsigned integers of the same order; 0: none
    for (int i = threadIdx.x & 31; i < n; i += 32) {
        const unsigned bits = __float_as_uint(v[i]);
        const unsigned k = ok[i] ? ((bits & 0x80000000u) ? ~bits : bits | 0x80000000u) : 0u;
        if (k > key) { key = k; at = i; }
    }
    const unsigned best = __reduce_max_sync(0xffffffffu, key);
    if (best == 0) return -1;
    return (int)__reduce_min_sync(0xffffffffu, key == best ? at : 0xffffffffu);
}

// four consecutive values as floats
__device__ __forceinline__ float4 four(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 four(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

// grid (ceil(tokens / kTok)): a CTA takes kTok neighbouring tokens, so that a row of W_r is read once for all of them; its warps
// share the rows, then warp k chooses for token k.  VEC: four columns at a time (width a multiple of 4, rows 16-byte aligned).
template <typename T, int kTok, bool VEC>
__global__ void __launch_bounds__(route_warps(kTok) * 32) moe_route_kernel(
        const T* __restrict__ h, const float* __restrict__ w_router, const float* __restrict__ correction,
        float* __restrict__ dense, int* __restrict__ chosen, float* __restrict__ chosen_w,
        float* __restrict__ id_weight, int tokens, int width, int n, int experts, int top,
        int groups, int keep, float scale, int sigmoid_scores, const float* __restrict__ bias, int pair_groups, int normalize,
        int gates) {
    __shared__ float zs[kTok][kRouteMax], cs[kTok][kRouteMax], gss[kTok][kRouteMax], shares[kTok][kRouteMax];
    __shared__ int pickeds[kTok][kRouteMax];
    __shared__ unsigned char oks[kTok][kRouteMax], goks[kTok][kRouteMax];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int first = blockIdx.x * kTok;
    const int nd = n + gates;                              // columns of the dense weights
    for (int e = warp; e < nd; e += route_warps(kTok)) {
        const float* wr = w_router + (size_t)e * width;
        float acc[kTok];
#pragma unroll
        for (int k = 0; k < kTok; ++k) acc[k] = 0.f;
        if (VEC) {
#pragma unroll 4
            for (int c = lane * 4; c < width; c += 128) {
                const float4 wv = four(wr + c);
#pragma unroll
                for (int k = 0; k < kTok; ++k) {
                    const float4 hv = four(h + (size_t)min(first + k, tokens - 1) * width + c);
                    acc[k] += (hv.x * wv.x + hv.y * wv.y) + (hv.z * wv.z + hv.w * wv.w);
                }
            }
        } else {
            for (int c = lane; c < width; c += 32) {
                const float wv = wr[c];
#pragma unroll
                for (int k = 0; k < kTok; ++k) acc[k] += to_f32(h[(size_t)min(first + k, tokens - 1) * width + c]) * wv;
            }
        }
#pragma unroll
        for (int k = 0; k < kTok; ++k) {
            const float a = warp_sum(acc[k]);
            if (lane == 0 && first + k < tokens) {
                if (e < n) zs[k][e] = a + (bias != nullptr ? bias[e] : 0.f);
                else dense[(size_t)(first + k) * nd + e] = 1.f / (1.f + expf(-a));
            }
        }
    }
    __syncthreads();
    const int t = first + warp;
    if (warp >= kTok || t >= tokens) return;
    float *z = zs[warp], *c = cs[warp], *gs = gss[warp], *share = shares[warp];
    int* picked = pickeds[warp];
    unsigned char *ok = oks[warp], *gok = goks[warp];
    const bool chosen_softmax = sigmoid_scores == 2;
    float mx = 0.f, sum = 1.f;
    if (sigmoid_scores == 0) {
        mx = -INFINITY;
        for (int e = lane; e < n; e += 32) mx = fmaxf(mx, z[e]);
        mx = warp_max(mx);
        sum = 0.f;
        for (int e = lane; e < n; e += 32) sum += expf(z[e] - mx);
        sum = warp_sum(sum);
    }
    __syncwarp();
    for (int e = lane; e < n; e += 32) {
        const float logit = z[e];
        const float s = chosen_softmax ? logit : (sigmoid_scores ? 1.f / (1.f + expf(-logit)) : expf(logit - mx) / sum);
        z[e] = s;
        // sigmoid scores without a correction are ranked by their logits: the same order, and two large logits do not
        // meet in a score that has rounded to 1
        c[e] = (sigmoid_scores && correction == nullptr) ? logit : s + (correction != nullptr ? correction[e] : 0.f);
        ok[e] = 0;
        dense[(size_t)t * nd + e] = 0.f;
    }
    __syncwarp();
    // the groups that stay: `keep` times the group whose best member (or best two) is largest (ties: the lower index)
    const int per = n / groups;
    for (int g = lane; g < groups; g += 32) {
        float gm = -INFINITY, second = -INFINITY;
        for (int i = 0; i < per; ++i) {
            const float v = c[g * per + i];
            if (v > gm) { second = gm; gm = v; }
            else second = fmaxf(second, v);
        }
        gs[g] = (pair_groups && per > 1) ? gm + second : gm;
        gok[g] = 1;
    }
    __syncwarp();
    for (int r = 0; r < keep; ++r) {
        const int best_g = warp_best(gs, gok, groups);
        if (best_g < 0) break;
        for (int i = lane; i < per; i += 32) ok[best_g * per + i] = 1;
        if (lane == 0) gok[best_g] = 0;
        __syncwarp();
    }
    // the `top` best of what stays: chosen_softmax weighs them by the softmax over their logits, the others by their scores
    float idw = 0.f, total = 0.f, best_all = 0.f;
    for (int r = 0; r < top; ++r) {
        const int e = warp_best(c, ok, n);
        float part = 0.f;
        if (e >= 0) {
            if (r == 0) best_all = c[e];
            part = chosen_softmax ? expf(c[e] - best_all) : z[e];
        }
        total += part;
        __syncwarp();
        if (lane == 0) {
            if (e >= 0) ok[e] = 0;
            chosen[(size_t)t * top + r] = e;
            picked[r] = e;
            share[r] = part;
        }
        __syncwarp();
    }
    const float factor = normalize ? scale / (total + 1e-20f) : scale;
    for (int r = lane; r < top; r += 32) {
        const int e = picked[r];
        const float wgt = e < 0 ? 0.f : (chosen_softmax ? share[r] / total * scale : share[r] * factor);
        chosen_w[(size_t)t * top + r] = wgt;
        if (e < 0) continue;
        dense[(size_t)t * nd + e] = wgt;
        if (e >= experts) idw += wgt;
    }
    idw = warp_sum(idw);
    if (lane == 0) id_weight[t] = idw;
}

extern "C" int lb_moe_route(const void* h, const float* w_router, const float* correction, float* dense, int* chosen,
                            float* chosen_w, float* id_weight, int tokens, int width, int n, int experts, int top, int groups,
                            int keep, float scale, int sigmoid_scores, const float* bias, int pair_groups, int normalize, int gates,
                            int dtype, void* stream) {
    if (tokens <= 0) return kOk;
    if (n <= 0 || experts < 0 || experts > n || top <= 0 || top > n || groups <= 0 || n % groups || keep <= 0 || keep > groups)
        return kBadSize;
    if (n > kRouteMax) return kTooLarge;
    if (sigmoid_scores < 0 || sigmoid_scores > 2 || gates < 0 || (sigmoid_scores == 2 && normalize)) return kBadSize;
    const bool vec = width % 4 == 0 && ((uintptr_t)h & 7) == 0 && ((uintptr_t)w_router & 15) == 0 && (dtype == kBF16 || ((uintptr_t)h & 15) == 0);
    const bool tile = tokens >= 4 * 148;                   // enough tokens for a CTA per four of them on every SM
#define LB_ROUTE(TOK, V) LB_DISPATCH_DTYPE(dtype, moe_route_kernel<T, TOK, V><<<(tokens + TOK - 1) / TOK, route_warps(TOK) * 32, 0, (cudaStream_t)stream>>>( \
        (const T*)h, w_router, correction, dense, chosen, chosen_w, id_weight, tokens, width, n, experts, top, groups, keep, scale, sigmoid_scores, bias, \
        pair_groups, normalize, gates))
    if (tile) { if (vec) { LB_ROUTE(4, true); } else { LB_ROUTE(4, false); } }
    else { if (vec) { LB_ROUTE(1, true); } else { LB_ROUTE(1, false); } }
#undef LB_ROUTE
    return launch_status();
}

enum : int { kClampedOutput = 0, kSiluInput = 1, kSiluOutput = 2, kGeluOutput = 3 };

__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

__device__ __forceinline__ float expert_act(float g, float u, float w, float limit, float act_alpha, int mode) {
    if (mode == kSiluInput) {
        const float wg = w * g;
        return wg / (1.f + expf(-wg)) * (w * u);
    }
    if (mode == kSiluOutput) return w * (g / (1.f + expf(-g)) * u);
    if (mode == kGeluOutput) return w * (gelu_tanh_f(g) * u);
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return w * (g / (1.f + expf(-act_alpha * g)) * (u + 1.f));
}

// gu: [T, experts, 2, ff] [2, tail_ff]; y: [T, experts, ff] [tail_ff]; dense: [T, n] (null: weight 1)
template <typename T>
__global__ void moe_activation_kernel(const T* __restrict__ gu, const float* __restrict__ dense, T* __restrict__ y,
                                      int experts, int ff, int n, float limit, float act_alpha, int mode, long in_stride,
                                      long out_stride, int tail_ff, int tail_gate) {
    const size_t t = blockIdx.z;
    const int e = blockIdx.y;
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    const bool tail = e == experts;
    const int size = tail ? tail_ff : ff;
    if (i >= size) return;
    const int col = tail ? tail_gate : e;
    const float w = (dense != nullptr && col >= 0) ? dense[t * n + col] : 1.f;
    float v = 0.f;
    if (w != 0.f) {
        const T* row = gu + t * in_stride + e * 2 * (size_t)ff;
        v = expert_act(to_f32(row[i]), to_f32(row[size + i]), w, limit, act_alpha, mode);
    }
    y[t * out_stride + e * (size_t)ff + i] = from_f32<T>(v);
}

// the same for bfloat16 rows with ff a multiple of 8: a CTA per token walks its experts' rows in 16-byte pieces, and writes
// zeros for the experts that were not chosen without reading their products
__global__ void __launch_bounds__(256) moe_activation_vec_kernel(const __nv_bfloat16* __restrict__ gu, const float* __restrict__ dense,
                                                                 __nv_bfloat16* __restrict__ y, int experts, int ff, int n,
                                                                 float limit, float act_alpha, int mode, long in_stride,
                                                                 long out_stride, int tail_ff, int tail_gate) {
    const size_t t = blockIdx.x;
    const int pieces = ff / 8, all = experts * pieces;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < all + tail_ff / 8; i += gridDim.y * blockDim.x) {
        const bool tail = i >= all;
        const int e = tail ? experts : i / pieces, pc = tail ? i - all : i % pieces;
        const int size = tail ? tail_ff : ff, col = tail ? tail_gate : e;
        const float w = (dense != nullptr && col >= 0) ? dense[t * n + col] : 1.f;
        uint4 out = make_uint4(0, 0, 0, 0);
        if (w != 0.f) {
            const __nv_bfloat16* row = gu + t * in_stride + e * 2 * (size_t)ff;
            const uint4 gv = *reinterpret_cast<const uint4*>(row + pc * 8);
            const uint4 uv = *reinterpret_cast<const uint4*>(row + size + pc * 8);
            const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
            const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
                if (mode == kSiluInput) {
                    const float g0 = w * g.x, g1 = w * g.y;
                    o2[k] = __floats2bfloat162_rn(__fdividef(g0, 1.f + __expf(-g0)) * (w * u.x), __fdividef(g1, 1.f + __expf(-g1)) * (w * u.y));
                } else if (mode == kSiluOutput) {
                    o2[k] = __floats2bfloat162_rn(w * (__fdividef(g.x, 1.f + __expf(-g.x)) * u.x), w * (__fdividef(g.y, 1.f + __expf(-g.y)) * u.y));
                } else if (mode == kGeluOutput) {
                    o2[k] = __floats2bfloat162_rn(w * (gelu_tanh_f(g.x) * u.x), w * (gelu_tanh_f(g.y) * u.y));
                } else {
                    const float g0 = fminf(g.x, limit), g1 = fminf(g.y, limit);
                    const float u0 = fminf(fmaxf(u.x, -limit), limit), u1 = fminf(fmaxf(u.y, -limit), limit);
                    o2[k] = __floats2bfloat162_rn(w * (g0 / (1.f + __expf(-act_alpha * g0)) * (u0 + 1.f)),
                                                  w * (g1 / (1.f + __expf(-act_alpha * g1)) * (u1 + 1.f)));
                }
            }
        }
        *reinterpret_cast<uint4*>(y + t * out_stride + e * (size_t)ff + pc * 8) = out;
    }
}

extern "C" int lb_moe_activation(const void* gu, const float* dense, void* y, int tokens, int experts, int ff, int n, float limit,
                                 float act_alpha, int mode, long in_stride, long out_stride, int tail_ff, int tail_gate, int dtype,
                                 void* stream) {
    if (tokens <= 0 || experts <= 0) return kOk;
    if (ff <= 0 || (dense != nullptr && n < experts) || experts > 65534 || mode < kClampedOutput || mode > kGeluOutput || tail_ff < 0
        || tail_gate >= n || in_stride < 2 * ((long)experts * ff + tail_ff) || out_stride < (long)experts * ff + tail_ff)
        return kBadSize;
    if (dtype == kBF16 && ff % 8 == 0 && tail_ff % 8 == 0 && (((uintptr_t)gu | (uintptr_t)y) & 15) == 0 && in_stride % 8 == 0 && out_stride % 8 == 0) {
        // few tokens: several CTAs share a token's columns
        const int pieces = (experts * ff + tail_ff) / 8;
        const int split = tokens >= 148 ? 1 : min(max(1, 296 / tokens), (pieces + 255) / 256);
        moe_activation_vec_kernel<<<dim3(tokens, split), 256, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)gu, dense, (__nv_bfloat16*)y, experts, ff,
                                                                          n, limit, act_alpha, mode, in_stride, out_stride, tail_ff, tail_gate);
        return launch_status();
    }
    dim3 grid((max(ff, tail_ff) + 127) / 128, experts + (tail_ff > 0), tokens);
    LB_DISPATCH_DTYPE(dtype, moe_activation_kernel<T><<<grid, 128, 0, (cudaStream_t)stream>>>(
        (const T*)gu, dense, (T*)y, experts, ff, n, limit, act_alpha, mode, in_stride, out_stride, tail_ff, tail_gate));
    return launch_status();
}

template <typename T>
__global__ void moe_add_identity_kernel(T* __restrict__ out, const T* __restrict__ h, const float* __restrict__ id_weight, int width) {
    const size_t t = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= width) return;
    const float w = id_weight[t];
    if (w != 0.f) out[t * width + c] = from_f32<T>(to_f32(out[t * width + c]) + w * to_f32(h[t * width + c]));
}

extern "C" int lb_moe_add_identity(void* out, const void* h, const float* id_weight, int tokens, int width, int dtype, void* stream) {
    if (tokens <= 0) return kOk;
    if (width <= 0) return kBadSize;
    dim3 grid((width + 255) / 256, tokens);
    LB_DISPATCH_DTYPE(dtype, moe_add_identity_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>((T*)out, (const T*)h, id_weight, width));
    return launch_status();
}

template <typename T>
__global__ void gelu_tanh_kernel(const T* __restrict__ in, T* __restrict__ out, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const float z = to_f32(in[i]);
    out[i] = from_f32<T>(0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))));
}

extern "C" int lb_gelu_tanh(const void* in, void* out, long n, int dtype, void* stream) {
    if (n <= 0) return kOk;
    LB_DISPATCH_DTYPE(dtype, gelu_tanh_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>((const T*)in, (T*)out, (size_t)n));
    return launch_status();
}

__device__ __forceinline__ float xielu_f(float z, float a, float b) {
    return z > 0.f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, expm1f(z) - z, 0.5f * z);
}

template <typename T>
__global__ void xielu_kernel(const T* __restrict__ in, T* __restrict__ out, const float* __restrict__ ab, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_f32<T>(xielu_f(to_f32(in[i]), ab[0], ab[1]));
}

// bfloat16, eight values (one 16-byte word) per thread
__global__ void xielu_vec_kernel(const uint4* __restrict__ in, uint4* __restrict__ out, const float* __restrict__ ab, size_t words) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= words) return;
    const float a = ab[0], b = ab[1];
    uint4 v = in[i];
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(p[e]); p[e] = __floats2bfloat162_rn(xielu_f(f.x, a, b), xielu_f(f.y, a, b)); }
    out[i] = v;
}

// ab: float32 [2], the factors a and b
extern "C" int lb_xielu(const void* in, void* out, const float* ab, long n, int dtype, void* stream) {
    if (n <= 0) return kOk;
    if (dtype == kBF16 && n % 8 == 0 && (((uintptr_t)in | (uintptr_t)out) & 15) == 0) {
        const size_t words = (size_t)n / 8;
        xielu_vec_kernel<<<(unsigned)((words + 255) / 256), 256, 0, (cudaStream_t)stream>>>((const uint4*)in, (uint4*)out, ab, words);
        return launch_status();
    }
    LB_DISPATCH_DTYPE(dtype, xielu_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>((const T*)in, (T*)out, ab, (size_t)n));
    return launch_status();
}

// x[t, c] <- silu(x[t, c] * scale[c]) for the first `cols` columns of every row (row stride in elements; scale may be null)
template <typename T>
__global__ void silu_columns_kernel(T* __restrict__ x, long stride, int cols, const float* __restrict__ scale, size_t total) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int c = (int)(i % cols);
    T* at = x + (i / cols) * stride + c;
    float v = to_f32(*at);
    if (scale != nullptr) v = round_to<T>(v * scale[c]);
    *at = from_f32<T>(silu_f(v));
}

extern "C" int lb_silu_columns(void* x, long stride, int rows, int cols, const float* scale, int dtype, void* stream) {
    if (rows <= 0 || cols <= 0) return kOk;
    if (stride < cols) return kBadSize;
    const size_t total = (size_t)rows * cols;
    LB_DISPATCH_DTYPE(dtype, silu_columns_kernel<T><<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>((T*)x, stride, cols, scale, total));
    return launch_status();
}
