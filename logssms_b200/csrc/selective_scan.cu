// Selective scan with a decay of its own for every (channel, state): the recurrence of Mamba's first form.
//
//   dt_t[c]   = softplus(w_t[c] + dt_bias[c])           w_t: the step's projection (32-bit, as handed in or made here)
//   S[c, n]  <- exp(dt_t[c] A[c, n]) S[c, n] + dt_t[c] x_t[c] B_t[n]            A = -exp(A_log); S float32
//   y_t[c]    = (sum_n S[c, n] C_t[n] + D[c] x_t[c]) * silu(z_t[c])             (uses the updated state)
//
// x, B, C and the gate z are activations; step size, decays, state and sums are float32 in every dtype.  The decays
// are exp2(dt * A log2(e)), one per (token, channel, state): the exponential unit bounds the kernel on long portions.
//
//  A CTA of 128 threads owns 128 / LN neighbouring channels of one request; LN lanes of a warp share a channel, each
//  with NPT neighbouring states in registers.  Tokens go through in blocks of TB: x, dt, z of the CTA's channels and the
//  block's B and C travel to registers while the block before is computed, then to shared memory, where the step
//  size, its product with x and D x are worked out once per (token, channel); the loop over the tokens touches shared
//  memory and registers only; the outputs leave through shared memory in rows of neighbouring channels.
//
//  selective_scan          : a request's tokens from its slot's state to its slot's state (a request that starts at
//                            position 0 starts from zeros whatever the slot holds).  With `dt_w` the step's
//                            low-rank projection rides along: w = dt_w low_t, the LN lanes of a channel sharing its row.
//  selective_scan_segments : long portions cut into segments that run side by side, two launches.  The first runs every
//                            request's first segment from the slot's state with its outputs, and every later segment
//                            but the last from zero, without outputs, leaving its end state and the sum of its step
//                            sizes (the product of its decays is exp(A * sum)).  In the second every later segment
//                            joins the segments before it into its start state and runs with outputs; the last one
//                            leaves the request's state in its slot.
#include "lb200/common.cuh"
using namespace lb200;

namespace {
constexpr int kThreads = 128;
constexpr float kLog2e = 1.4426950408889634f;

struct ScanArgs {
    const void* x; long x_stride;          // [tokens, inner] view
    const float* w;                        // [tokens, inner] the step's projection, or null: made from `low` and `dt_w`
    const void* low; long low_stride;      // [tokens, rank + 2 * n] view: low-rank step | B | C
    const void* dt_w;                      // [inner, rank]
    const float* dt_bias; const float* A_log; const float* D;
    const void* gate; long gate_stride;    // z: [tokens, inner] view
    float* state;                          // [slots, inner, n]
    void* y;                               // [tokens, inner]
    const int* cu; const int* start_pos; const int* slots;
    const int* list;                       // requests to run, or (segments) int32 [items, 4]
    int inner, n, rank;
    int seg_tokens; float* seg_state; float* seg_dt;
};

__device__ __forceinline__ float ex2(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// PASS 0: whole portions; 1, 2: the two launches over segments
template <typename T, int LN, int NPT, int TB, int PASS>
__global__ void __launch_bounds__(kThreads) selective_scan_kernel(ScanArgs a) {
    constexpr int CH = kThreads / LN, NP = LN * NPT;
    constexpr int KX = (TB * CH + kThreads - 1) / kThreads, KB = (TB * 2 * NP + kThreads - 1) / kThreads;
    __shared__ __align__(16) float Bs[TB][NP], Cs[TB][NP];
    __shared__ float dts[TB][CH], us[TB][CH], ys[TB][CH];
    const int ch = threadIdx.x / LN, ln = threadIdx.x % LN;
    const int c0 = blockIdx.x * CH, c = c0 + ch;
    const bool c_ok = c < a.inner;
    int b, first, last, seg = 0;
    bool with_out = true, last_seg = true;
    if (PASS == 0) {
        b = a.list != nullptr ? a.list[blockIdx.y] : blockIdx.y;
        if (b < 0) return;
        first = a.cu[b];
        last = a.cu[b + 1];
    } else {
        b = a.list[4 * blockIdx.y];
        if (b < 0) return;
        const int t0 = a.list[4 * blockIdx.y + 3], begin = a.cu[b], len = a.cu[b + 1] - begin;
        seg = t0 / a.seg_tokens;
        last_seg = t0 + a.seg_tokens >= len;
        if (PASS == 1 ? (seg > 0 && last_seg) : seg == 0) return;
        first = begin + t0;
        last = begin + min(len, t0 + a.seg_tokens);
        with_out = PASS == 2 || seg == 0;
    }
    if (first >= last) return;
    // the thread's decay rates and states, as 16-byte pieces where the state size fills the lanes exactly; the rates are worked
    // out after the first block's loads are on their way too
    float A2[NPT], S[NPT];
    const bool full = a.n == NP && (((uintptr_t)a.A_log | (uintptr_t)a.state) & 15) == 0;
    auto load_states = [&](const float* row, float (&out)[NPT]) {
        if (full) {
#pragma unroll
            for (int i = 0; i < NPT; i += 4) {
                const float4 v = *reinterpret_cast<const float4*>(row + ln * NPT + i);
                out[i] = v.x; out[i + 1] = v.y; out[i + 2] = v.z; out[i + 3] = v.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < NPT; ++i) out[i] = ln * NPT + i < a.n ? row[ln * NPT + i] : 0.f;
        }
    };
#pragma unroll
    for (int i = 0; i < NPT; ++i) A2[i] = S[i] = 0.f;
    if (c_ok) load_states(a.A_log + (size_t)c * a.n, A2);
    float* slot_state = a.state + ((size_t)a.slots[b] * a.inner + (c_ok ? c : 0)) * a.n;
    if (PASS != 2 && seg == 0 && a.start_pos[b] > 0 && c_ok) load_states(slot_state, S);
    const T* x = (const T*)a.x;
    const T* low = (const T*)a.low;
    const T* gate = (const T*)a.gate;
    // the element of a block that this thread stages: token threadIdx.x / CH (+ kThreads / CH per turn), channel cl
    constexpr int TSTEP = kThreads / CH;
    const int tl = threadIdx.x / CH, cl = threadIdx.x % CH;
    const bool cl_ok = c0 + cl < a.inner;
    const float cl_bias = cl_ok ? a.dt_bias[c0 + cl] : 0.f, cl_D = cl_ok ? a.D[c0 + cl] : 0.f;
    // (raw values: converting them here would wait for them here)
    T rx[KX], rz[KX], rb[KB];
    float rw[KX];
    const T zero = from_f32<T>(0.f);
    auto fetch = [&](int t0) {
        const int nt = min(TB, last - t0);
#pragma unroll
        for (int k = 0; k < KX; ++k) {
            const int t = tl + k * TSTEP;
            rx[k] = rz[k] = zero;
            rw[k] = 0.f;
            if (t < nt && cl_ok) {
                rx[k] = x[(size_t)(t0 + t) * a.x_stride + c0 + cl];
                if (a.w != nullptr) rw[k] = a.w[(size_t)(t0 + t) * a.inner + c0 + cl];
                if (with_out) rz[k] = gate[(size_t)(t0 + t) * a.gate_stride + c0 + cl];
            }
        }
#pragma unroll
        for (int k = 0; k < KB; ++k) {
            const int i = threadIdx.x + k * kThreads, t = i / (2 * NP), r = i % (2 * NP);
            const int s = r < NP ? r : r - NP;
            rb[k] = (t < nt && s < a.n) ? low[(size_t)(t0 + t) * a.low_stride + a.rank + (r < NP ? 0 : a.n) + s] : zero;
        }
    };
    fetch(first);
#pragma unroll
    for (int i = 0; i < NPT; ++i) A2[i] = (c_ok && ln * NPT + i < a.n) ? -expf(A2[i]) * kLog2e : 0.f;
    if (PASS == 2 && c_ok) {
        // the segments before this one, joined in order (the first one's end state holds what the slot held)
        for (int g = 0; g < seg; ++g) {
            const size_t item = blockIdx.y - seg + g;
            const float sum = g == 0 ? 0.f : a.seg_dt[item * a.inner + c];
            float e[NPT];
            load_states(a.seg_state + (item * a.inner + c) * a.n, e);
#pragma unroll
            for (int i = 0; i < NPT; ++i) S[i] = ex2(sum * A2[i]) * S[i] + e[i];
        }
    }
    float dt_sum = 0.f;
    for (int t0 = first; t0 < last; t0 += TB) {
        const int nt = min(TB, last - t0);
        __syncthreads();                                   // the block before has left shared memory
        if (a.w == nullptr) {
            // w = dt_w low: the lanes of a channel share its row of dt_w, in pieces of 16 bytes where they are aligned
            constexpr int E = 16 / sizeof(T);
            const bool pieces = a.rank % E == 0 && a.low_stride % E == 0 && (((uintptr_t)a.dt_w | (uintptr_t)a.low) & 15) == 0;
            for (int t = 0; t < nt; ++t) {
                float acc = 0.f;
                const T* wr = (const T*)a.dt_w + (size_t)(c_ok ? c : 0) * a.rank;
                const T* lr = low + (size_t)(t0 + t) * a.low_stride;
                if (c_ok) {
                    if (pieces) {
#pragma unroll 4
                        for (int r = ln * E; r < a.rank; r += LN * E) {
                            const uint4 wv = *reinterpret_cast<const uint4*>(wr + r), lv = *reinterpret_cast<const uint4*>(lr + r);
                            const T *we = reinterpret_cast<const T*>(&wv), *le = reinterpret_cast<const T*>(&lv);
#pragma unroll
                            for (int e = 0; e < E; ++e) acc += to_f32(we[e]) * to_f32(le[e]);
                        }
                    } else {
                        for (int r = ln; r < a.rank; r += LN) acc += to_f32(wr[r]) * to_f32(lr[r]);
                    }
                }
#pragma unroll
                for (int off = 1; off < LN; off <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
                if (ln == 0) dts[t][ch] = acc;
            }
            __syncthreads();
        }
#pragma unroll
        for (int k = 0; k < KX; ++k) {
            const int t = tl + k * TSTEP;
            if (t < TB) {
                const float xv = to_f32(rx[k]);
                const float dt = (t < nt && cl_ok) ? softplus_f((a.w != nullptr ? rw[k] : dts[t][cl]) + cl_bias) : 0.f;
                dts[t][cl] = dt;
                us[t][cl] = dt * xv;
                ys[t][cl] = cl_D * xv;
            }
        }
#pragma unroll
        for (int k = 0; k < KB; ++k) {
            const int i = threadIdx.x + k * kThreads, t = i / (2 * NP), r = i % (2 * NP);
            if (t < TB) {
                if (r < NP) Bs[t][r] = to_f32(rb[k]);
                else Cs[t][r - NP] = to_f32(rb[k]);
            }
        }
        float z[KX];
#pragma unroll
        for (int k = 0; k < KX; ++k) z[k] = to_f32(rz[k]);
        if (t0 + TB < last) fetch(t0 + TB);
        __syncthreads();
        // one token for this thread's states: its share of the output sum
        auto step = [&](int t) {
            const float dt = dts[t][ch], u = us[t][ch];
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < NPT; i += 4) {
                const float4 bv = *reinterpret_cast<const float4*>(&Bs[t][ln * NPT + i]);
                const float4 cv = *reinterpret_cast<const float4*>(&Cs[t][ln * NPT + i]);
                S[i] = ex2(dt * A2[i]) * S[i] + u * bv.x;
                S[i + 1] = ex2(dt * A2[i + 1]) * S[i + 1] + u * bv.y;
                S[i + 2] = ex2(dt * A2[i + 2]) * S[i + 2] + u * bv.z;
                S[i + 3] = ex2(dt * A2[i + 3]) * S[i + 3] + u * bv.w;
                acc += S[i] * cv.x + S[i + 1] * cv.y + S[i + 2] * cv.z + S[i + 3] * cv.w;
            }
            return acc;
        };
        if (with_out) {
            if (nt == 1) {
                float acc = step(0);
#pragma unroll
                for (int off = 1; off < LN; off <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
                if (ln == 0) ys[0][ch] += acc;
            } else {
                // G tokens at a time, their sums over the LN lanes taken together: at every halving a lane keeps one half of
                // the tokens and hands the other half over, so that lane g (mod G) ends with token g's sum.  (Tokens behind the
                // last one have dt = 0 and zero inputs: they change nothing.)
                constexpr int G = LN < TB ? LN : TB;
                for (int g0 = 0; g0 < nt; g0 += G) {
                    float acc[G];
#pragma unroll
                    for (int g = 0; g < G; ++g) acc[g] = step(g0 + g);
#pragma unroll
                    for (int off = G / 2; off > 0; off >>= 1) {
                        const bool upper = ln & off;
#pragma unroll
                        for (int g = 0; g < off; ++g) {
                            const float mine = upper ? acc[g + off] : acc[g], other = upper ? acc[g] : acc[g + off];
                            acc[g] = mine + __shfl_xor_sync(0xffffffffu, other, off);
                        }
                    }
#pragma unroll
                    for (int off = G; off < LN; off <<= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], off);
                    if (ln < G) ys[g0 + ln][ch] += acc[0];
                }
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < KX; ++k) {
                const int t = tl + k * TSTEP;
                if (t < nt && cl_ok)
                    ((T*)a.y)[(size_t)(t0 + t) * a.inner + c0 + cl] = from_f32<T>(ys[t][cl] * (sizeof(T) == 2 ? silu_fast(z[k]) : silu_f(z[k])));
            }
        } else {
#pragma unroll 4
            for (int t = 0; t < nt; ++t) {
                const float dt = dts[t][ch], u = us[t][ch];
                dt_sum += dt;
#pragma unroll
                for (int i = 0; i < NPT; i += 4) {
                    const float4 bv = *reinterpret_cast<const float4*>(&Bs[t][ln * NPT + i]);
                    S[i] = ex2(dt * A2[i]) * S[i] + u * bv.x;
                    S[i + 1] = ex2(dt * A2[i + 1]) * S[i + 1] + u * bv.y;
                    S[i + 2] = ex2(dt * A2[i + 2]) * S[i + 2] + u * bv.z;
                    S[i + 3] = ex2(dt * A2[i + 3]) * S[i + 3] + u * bv.w;
                }
            }
        }
    }
    if (!c_ok) return;
    float* dst = slot_state;
    if (PASS == 1 && !last_seg) {
        dst = a.seg_state + ((size_t)blockIdx.y * a.inner + c) * a.n;
        if (ln == 0) a.seg_dt[(size_t)blockIdx.y * a.inner + c] = dt_sum;
    } else if (PASS == 2 && !last_seg) {
        return;
    }
    if (full) {
#pragma unroll
        for (int i = 0; i < NPT; i += 4) *reinterpret_cast<float4*>(dst + ln * NPT + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < NPT; ++i) if (ln * NPT + i < a.n) dst[ln * NPT + i] = S[i];
    }
}

template <typename T, int LN, int NPT, int TB>
int launch_sized(const ScanArgs& a, int items, bool segmented, cudaStream_t st) {
    constexpr int CH = kThreads / LN;
    dim3 grid((a.inner + CH - 1) / CH, items);
    if (!segmented) {
        selective_scan_kernel<T, LN, NPT, TB, 0><<<grid, kThreads, 0, st>>>(a);
        return launch_status();
    }
    selective_scan_kernel<T, LN, NPT, TB, 1><<<grid, kThreads, 0, st>>>(a);
    const int rc = launch_status();
    if (rc != 0) return rc;
    selective_scan_kernel<T, LN, NPT, TB, 2><<<grid, kThreads, 0, st>>>(a);
    return launch_status();
}

template <typename T>
int launch(const ScanArgs& a, int items, bool segmented, cudaStream_t st) {
    if (a.n <= 4) return launch_sized<T, 1, 4, 4>(a, items, segmented, st);
    if (a.n <= 8) return launch_sized<T, 2, 4, 8>(a, items, segmented, st);
    if (a.n <= 16) return launch_sized<T, 4, 4, 16>(a, items, segmented, st);
    if (a.n <= 32) return launch_sized<T, 8, 4, 16>(a, items, segmented, st);
    if (a.n <= 64) return launch_sized<T, 8, 8, 16>(a, items, segmented, st);
    if (a.n <= 128) return launch_sized<T, 16, 8, 8>(a, items, segmented, st);
    if (a.n <= 256) return launch_sized<T, 32, 8, 8>(a, items, segmented, st);
    return kTooLarge;
}

bool sizes_ok(const ScanArgs& a) {
    return a.inner > 0 && a.n > 0 && a.rank >= 0 && a.x_stride >= a.inner && a.gate_stride >= a.inner && a.low_stride >= a.rank + 2 * (long)a.n
           && (a.w != nullptr || a.dt_w != nullptr);
}
}  // namespace

// w: float32 [tokens, inner] (the step's projection without its bias), or null with dt_w [inner, rank] in the activation
// dtype; state sizes up to 256; `requests` counts `list` (int32 request indices, -1: nothing) or, without a list, the batch.
extern "C" int lb_selective_scan(const void* x, long x_stride, const float* w, const void* low, long low_stride, const void* dt_w,
                                 const float* dt_bias, const float* A_log, const float* D, const void* gate, long gate_stride,
                                 float* state, void* y, const int* cu, const int* start_pos, const int* slots, const int* list,
                                 int requests, int inner, int n, int rank, int dtype, void* stream) {
    if (requests <= 0) return kOk;
    ScanArgs a{x, x_stride, w, low, low_stride, dt_w, dt_bias, A_log, D, gate, gate_stride, state, y, cu, start_pos, slots, list,
               inner, n, rank, 0, nullptr, nullptr};
    if (!sizes_ok(a) || requests > 65535) return kBadSize;
    LB_DISPATCH_DTYPE(dtype, return launch<T>(a, requests, false, (cudaStream_t)stream));
    return kOk;
}

// segments: int32 [items, 4] (request, -, -, first token within its portion), a request's segments of seg_tokens tokens one
// after the other; request -1: nothing.  seg_state: float32 scratch [items, inner, n]; seg_dt: float32 scratch [items, inner].
extern "C" int lb_selective_scan_segments(const void* x, long x_stride, const float* w, const void* low, long low_stride,
                                          const float* dt_bias, const float* A_log, const float* D, const void* gate, long gate_stride,
                                          float* state, void* y, const int* cu, const int* start_pos, const int* slots,
                                          const int* segments, int items, int seg_tokens, float* seg_state, float* seg_dt, int inner,
                                          int n, int rank, int dtype, void* stream) {
    if (items <= 0) return kOk;
    ScanArgs a{x, x_stride, w, low, low_stride, nullptr, dt_bias, A_log, D, gate, gate_stride, state, y, cu, start_pos, slots, segments,
               inner, n, rank, seg_tokens, seg_state, seg_dt};
    if (!sizes_ok(a) || items > 65535 || seg_tokens <= 0) return kBadSize;
    LB_DISPATCH_DTYPE(dtype, return launch<T>(a, items, true, (cudaStream_t)stream));
    return kOk;
}
