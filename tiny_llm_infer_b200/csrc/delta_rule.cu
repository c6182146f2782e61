// The delta rule with a decay per head and key channel, as a recurrence over a state S [dk, dv] per
// (request, head) that lives in float32 and is carried from step to step:
//
//   S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t.
//
// Three kernels serve a step, prompt portions and single tokens alike:
//
//   delta_prepare  one block per token: the short causal convolution of the q, k and v channels (taps
//                  reaching before the portion come from the request's state), SiLU, unit length of q
//                  and k per head (q times a scale), g = exp(-rate_h softplus(a + bias)) and
//                  beta = sigmoid(b); all results in float32.
//   delta_scan     one block per (portion, head, group of value columns): a column of S is independent of
//                  the others, so a thread keeps a slice of one column in registers (the dk rows are dealt
//                  to R neighbouring lanes, which add their partial dot products with shuffles) and walks
//                  the portion's tokens, which come through two stages of shared memory sixteen at a time
//                  (cp.async: the next sixteen are on their way while these are walked; eight for the widest keys).
//   delta_finish   one block per token: o divided by its root mean square per head, times a weight, times
//                  sigmoid(gate); the block of a portion's last token also moves the convolution's
//                  window of the request's state on.
//
// State of a request: [heads][per][dv][R] floats of S (row i = r * per + il; rows past dk stay zero), then
// [taps - 1][channels] inputs of the convolution, the newest last.  R and per follow from dk alone
// (`tllm_delta_rule_lanes`), so every step of a request finds the layout the last one left.
#include "common.cuh"

namespace tllm {

constexpr int kScanMaxPer = 16;     // rows of a column that one thread keeps

// Tokens staged at a time: sixteen, eight where 32 lanes share a column (the widest keys), whose rows would not fit.
__host__ __device__ constexpr int scan_chunk(int lanes) { return lanes >= 32 ? 8 : 16; }

static inline int delta_lanes(int dk) {
    int r = 4;
    while (r < 32 && (dk + r - 1) / r > kScanMaxPer) r *= 2;
    return r;
}

__device__ __forceinline__ float softplus_f32(float x) {
    return x > 20.0f ? x : log1pf(expf(x));
}

// ---------------------------------------------------------------- prepare
template <typename T>
__global__ void delta_prepare_kernel(const T* proj, int ld, const T* __restrict__ conv_w, int taps,
                                     const float* a, int lda, const float* __restrict__ dt_bias,
                                     const float* __restrict__ rate, const int* __restrict__ token_slot,
                                     const float* state, long long state_stride, long long tail_off,
                                     int heads, int kv_heads, int dk, int dv, float q_scale, float unit_eps,
                                     float* qn, float* kn, float* vv, float* decay, float* beta, int n_rows,
                                     int decay_per_head, int beta_col) {
    extern __shared__ float y[];                 // [channels] after convolution and SiLU
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;
    const int qk = kv_heads * dk, channels = 2 * qk + heads * dv;
    int back = 0;                                // rows before this one that belong to the same portion
    for (int j = 1; j < taps; ++j) {
        if (t - j >= 0 && token_slot[t - j] == slot) back = j;
        else break;
    }
    const float* tail = state + (long long)slot * state_stride + tail_off;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
        float acc = 0.0f;
        for (int j = 0; j < taps; ++j) {
            const float w = to_f32<T>(conv_w[(size_t)c * taps + (taps - 1 - j)]);
            float x;
            if (j <= back) x = to_f32<T>(proj[(size_t)(t - j) * ld + c]);
            else x = tail[(size_t)(taps - 1 - (j - back)) * channels + c];
            acc += w * x;
        }
        y[c] = acc / (1.0f + expf(-acc));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int u = warp; u < 2 * kv_heads; u += warps) {          // q heads, then k heads
        const float* src = y + (size_t)u * dk;
        float sum = 0.0f;
        for (int e = lane; e < dk; e += 32) sum += src[e] * src[e];
        sum = warp_sum(sum);
        const bool is_q = u < kv_heads;
        const float sc = (is_q ? q_scale : 1.0f) / sqrtf(sum + unit_eps);
        float* dst = is_q ? qn + (size_t)t * qk + (size_t)u * dk : kn + (size_t)t * qk + (size_t)(u - kv_heads) * dk;
        for (int e = lane; e < dk; e += 32) dst[e] = src[e] * sc;
    }
    for (int e = threadIdx.x; e < heads * dv; e += blockDim.x) vv[(size_t)t * heads * dv + e] = y[2 * qk + e];
    for (int e = threadIdx.x; e < heads * dk; e += blockDim.x) {
        const int ai = decay_per_head ? e / dk : e;          // one decay per head serves all its key channels
        const float x = a[(size_t)t * lda + ai] + dt_bias[ai];
        decay[(size_t)t * heads * dk + e] = expf(-rate[e / dk] * softplus_f32(x));
    }
    for (int h = threadIdx.x; h < heads; h += blockDim.x) {
        const float b = to_f32<T>(proj[(size_t)t * ld + beta_col + h]);
        beta[(size_t)t * heads + h] = 1.0f / (1.0f + expf(-b));
    }
}

// 8-element accesses of either storage type (the convolution's inputs and taps), and of float32
template <typename T> struct Ld8;
template <> struct Ld8<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[8]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
};
template <> struct Ld8<bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[8]) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[8]) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};

// The same with eight channels per thread and access (rows of proj, the taps as [taps][channels], dk and dv
// multiples of eight, everything on 16-byte boundaries).
// TAPS: the number of taps if it is 2, 3 or 4 (their loads are then all issued before the first product), 0 for
// any other number.
template <typename T, int TAPS>
__global__ void delta_prepare_vec_kernel(const T* proj, int ld, const T* __restrict__ conv_t, int taps,
                                         const float* a, int lda, const float* __restrict__ dt_bias,
                                         const float* __restrict__ rate, const int* __restrict__ token_slot,
                                         const float* state, long long state_stride, long long tail_off,
                                         int heads, int kv_heads, int dk, int dv, float q_scale, float unit_eps,
                                         float* qn, float* kn, float* vv, float* decay, float* beta, int n_rows,
                                         int decay_per_head, int beta_col) {
    extern __shared__ __align__(16) float y[];   // [2 * kv_heads * dk] q and k after convolution and SiLU
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;
    const int qk = kv_heads * dk, channels = 2 * qk + heads * dv;
    int back = 0;
    for (int j = 1; j < taps; ++j) {
        if (t - j >= 0 && token_slot[t - j] == slot) back = j;
        else break;
    }
    const float* tail = state + (long long)slot * state_stride + tail_off;
    // With few rows a token's work is dealt to gridDim.y blocks: whole q and k heads (their norms need the
    // head together), an even share of the v channels, of the decays, and the betas to the first.
    const int Y = gridDim.y, yb = blockIdx.y;
    const int u0 = (2 * kv_heads * yb) / Y, u1 = (2 * kv_heads * (yb + 1)) / Y;         // q heads, then k heads
    const int vc = heads * dv / 8, v0 = 2 * qk + (vc * yb / Y) * 8, v1 = 2 * qk + (vc * (yb + 1) / Y) * 8;
    auto conv8 = [&](int c, float (&acc)[8]) {
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = 0.0f;
        if (TAPS > 0) {
            float w[TAPS > 0 ? TAPS : 1][8], x[TAPS > 0 ? TAPS : 1][8];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                Ld8<T>::load(conv_t + (size_t)(TAPS - 1 - j) * channels + c, w[j]);
                if (j <= back) Ld8<T>::load(proj + (size_t)(t - j) * ld + c, x[j]);
                else Ld8<float>::load(tail + (size_t)(TAPS - 1 - (j - back)) * channels + c, x[j]);
            }
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] += w[j][e] * x[j][e];
        } else {
            for (int j = 0; j < taps; ++j) {
                float w[8], x[8];
                Ld8<T>::load(conv_t + (size_t)(taps - 1 - j) * channels + c, w);
                if (j <= back) Ld8<T>::load(proj + (size_t)(t - j) * ld + c, x);
                else Ld8<float>::load(tail + (size_t)(taps - 1 - (j - back)) * channels + c, x);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] += w[e] * x[e];
            }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = acc[e] / (1.0f + expf(-acc[e]));
    };
    for (int c = u0 * dk + threadIdx.x * 8; c < u1 * dk; c += blockDim.x * 8) {
        float acc[8];
        conv8(c, acc);
        Ld8<float>::store(y + (c - u0 * dk), acc);
    }
    for (int c = v0 + threadIdx.x * 8; c < v1; c += blockDim.x * 8) {
        float acc[8];
        conv8(c, acc);
        Ld8<float>::store(vv + (size_t)t * heads * dv + (c - 2 * qk), acc);
    }
    const int dq = heads * dk / 4, e0 = (dq * yb / Y) * 4, e1 = (dq * (yb + 1) / Y) * 4;
    for (int e = e0 + threadIdx.x * 4; e < e1; e += blockDim.x * 4) {
        float4 x, b;
        if (decay_per_head) {                        // dk is a multiple of eight: the four share a head
            const float xa = a[(size_t)t * lda + e / dk], xb = dt_bias[e / dk];
            x = make_float4(xa, xa, xa, xa);
            b = make_float4(xb, xb, xb, xb);
        } else {
            x = *reinterpret_cast<const float4*>(a + (size_t)t * lda + e);
            b = *reinterpret_cast<const float4*>(dt_bias + e);
        }
        const float rt = rate[e / dk];
        float4 g;
        g.x = expf(-rt * softplus_f32(x.x + b.x)); g.y = expf(-rt * softplus_f32(x.y + b.y));
        g.z = expf(-rt * softplus_f32(x.z + b.z)); g.w = expf(-rt * softplus_f32(x.w + b.w));
        *reinterpret_cast<float4*>(decay + (size_t)t * heads * dk + e) = g;
    }
    if (yb == 0)
        for (int h = threadIdx.x; h < heads; h += blockDim.x) {
            const float b = to_f32<T>(proj[(size_t)t * ld + beta_col + h]);
            beta[(size_t)t * heads + h] = 1.0f / (1.0f + expf(-b));
        }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int u = u0 + warp; u < u1; u += warps) {
        const float* src = y + (size_t)(u - u0) * dk;
        float sum = 0.0f;
        for (int e = lane * 4; e < dk; e += 128) {
            const float4 v = *reinterpret_cast<const float4*>(src + e);
            sum += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        sum = warp_sum(sum);
        const bool is_q = u < kv_heads;
        const float sc = (is_q ? q_scale : 1.0f) / sqrtf(sum + unit_eps);
        float* dst = is_q ? qn + (size_t)t * qk + (size_t)u * dk : kn + (size_t)t * qk + (size_t)(u - kv_heads) * dk;
        for (int e = lane * 4; e < dk; e += 128) {
            float4 v = *reinterpret_cast<const float4*>(src + e);
            v.x *= sc; v.y *= sc; v.z *= sc; v.w *= sc;
            *reinterpret_cast<float4*>(dst + e) = v;
        }
    }
}

// ---------------------------------------------------------------- scan
template <int R>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = R / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ void cp_async_f32(float* dst, const float* src, bool valid) {
    const int bytes = valid ? 4 : 0;                 // zero fill where there is nothing to read
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void cp_async_f32x4(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// A lane r of a column keeps the rows i = r * per + il, il < per, as PER registers; in shared memory a token's
// k (and q, g) row is laid out [R][PER + 4]: a lane's rows are neighbours, so it reads them four at a time, and
// the four floats between the lanes' runs keep those reads off each other's banks.
template <int R, int PER, int VECS>
struct ScanLayout {
    static constexpr int kChunk = scan_chunk(R);
    static constexpr int kRow = R * (PER + 4);                               // floats of one token's k (or q, g, e) row
    __host__ __device__ static constexpr int stage_floats(int cols) {       // k, q, g (, e), the value columns, the betas, the keeps
        return (kChunk * (VECS * kRow + cols + 2) + 3) / 4 * 4;
    }
};

// R lanes share a column, each keeps PER rows of it at most.  A thread takes NC neighbouring columns (one, or two in
// steps of long portions): it reads a token's rows from shared memory once for all of them, and those reads are what a
// long portion's time goes with.  A column's arithmetic is the same either way.  The chunks of tokens come through two stages
// filled by cp.async, so that the next chunk is on its way while this one is walked.  A token's step, per
// thread: S <- g S, dot = sum S k, u = beta (v - dot), S <- S + k u, o = sum S q.  Only S is carried from token
// to token; the read-out's sum is off that path.
//
// MODE picks the recurrence.  kScanDelta: the delta rule above.  kScanPlain: no correction, S <- g S + k (b v)^T with
// the write strength b (one where `beta` is null).  kScanMemory: a matrix memory whose two gates come as logarithms
// (`beta` the write's, `fgate` the keep's) and are held under a running maximum m kept per column in the request's
// state at `aux_off`: m' = max(f + m, i), S <- exp(f + m - m') S + exp(i - m') k v^T; its last value column is the
// normaliser (the prepare kernel feeds it ones), whose read-out leaves as max(|n . q|, exp(-m')) + floor_eps in
// `den` while the other columns go to o_raw [., heads, dv - 1].  kScanHeadDecay: kScanPlain with one decay per
// (token, head) for all rows of S and a write strength likewise, S <- a S + k (w v)^T; the decays come in `beta`
// [., heads], the strengths in `fgate` [., heads], and `decay` is not read.  kScanErase: a delta rule whose removal has
// a rate per key channel and reads the state before its decay, S <- g S - e (k^T S)^T + k v^T with k the unit key and
// e = rate * k in `erase` (v comes already multiplied by the key's length); no beta.  kScanFixedDecay: no correction, and one
// decay per head that no token changes, S <- a_h S + k v^T, the a_h in `fgate` [heads]; neither `decay` nor `beta` are read.
enum ScanMode : int { kScanDelta = 0, kScanPlain = 1, kScanMemory = 2, kScanHeadDecay = 3, kScanErase = 4, kScanFixedDecay = 5 };
__host__ __device__ constexpr int scan_vecs(int mode) { return mode == kScanErase ? 4 : 3; }

template <int R, int PER, int MODE, int NC>
__global__ void __launch_bounds__(NC == 1 ? 256 : 128, 2)
delta_scan_kernel(const int* __restrict__ seg_info, const int* __restrict__ token_slot,
                  const float* qn, const float* kn, const float* vv, const float* decay,
                  const float* beta, float* state, long long state_stride, int heads,
                  int kv_heads, int dk, int dv, int cols, int vec, float* o_raw,
                  const float* fgate, const float* erase, long long aux_off, float floor_eps, float* den) {
    extern __shared__ __align__(16) float sm[];
    using L = ScanLayout<R, PER, scan_vecs(MODE)>;
    constexpr int kScanChunk = L::kChunk;
    constexpr bool kDecayRows = MODE == kScanDelta || MODE == kScanPlain || MODE == kScanErase;
    constexpr int kLane = PER + 4;
    TLLM_PDL_ENTER();
    const int seg = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * cols;
    int slot, start, len;
    if (seg_info != nullptr) {
        slot = seg_info[4 * seg]; start = seg_info[4 * seg + 1]; len = seg_info[4 * seg + 2];
    } else {
        slot = token_slot[seg]; start = seg; len = 1;
    }
    if (slot < 0 || len <= 0) return;
    const int per = (dk + R - 1) / R;
    const int r = threadIdx.x % R, jl = threadIdx.x / R * NC;  // lane of the columns, the first of them in the block
    const int j = col0 + jl;
    const int kvh = head / (heads / kv_heads);
    const int stage_floats = L::stage_floats(cols);
    float* o_s = sm + 2 * stage_floats;               // [chunk][cols]
    // rows that no copy writes (past per in a lane, past dk in the last lanes) are zeros: they add nothing
    if (per < PER || dk < R * per) {
        for (int i = threadIdx.x; i < 2 * stage_floats; i += blockDim.x) sm[i] = 0.0f;
        __syncthreads();
    }

    auto issue = [&](int c0, int st) {
        const int n = min(kScanChunk, len - c0);
        float* k_s = sm + st * stage_floats;
        float* q_s = k_s + kScanChunk * L::kRow;
        float* g_s = q_s + kScanChunk * L::kRow;
        float* e_s = g_s + kScanChunk * L::kRow;
        float* v_s = e_s + (MODE == kScanErase ? kScanChunk * L::kRow : 0);
        float* b_s = v_s + kScanChunk * cols;
        float* f_s = b_s + kScanChunk;
        if (vec) {                                    // dk and per multiples of four: four rows of one lane at a time
            const int quads = dk >> 2;
            for (int i = threadIdx.x; i < n * quads; i += blockDim.x) {
                const int tt = i / quads, e = (i - tt * quads) * 4;
                const int at = tt * L::kRow + (e / per) * kLane + e % per;
                const size_t row = (size_t)(start + c0 + tt);
                cp_async_f32x4(k_s + at, kn + (row * kv_heads + kvh) * dk + e);
                cp_async_f32x4(q_s + at, qn + (row * kv_heads + kvh) * dk + e);
                if (kDecayRows) cp_async_f32x4(g_s + at, decay + (row * heads + head) * dk + e);
                if (MODE == kScanErase) cp_async_f32x4(e_s + at, erase + (row * heads + head) * dk + e);
            }
        } else {
            for (int i = threadIdx.x; i < n * dk; i += blockDim.x) {
                const int tt = i / dk, e = i - tt * dk;
                const int at = tt * L::kRow + (e / per) * kLane + e % per;
                const size_t row = (size_t)(start + c0 + tt);
                cp_async_f32(k_s + at, kn + (row * kv_heads + kvh) * dk + e, true);
                cp_async_f32(q_s + at, qn + (row * kv_heads + kvh) * dk + e, true);
                if (kDecayRows) cp_async_f32(g_s + at, decay + (row * heads + head) * dk + e, true);
                if (MODE == kScanErase) cp_async_f32(e_s + at, erase + (row * heads + head) * dk + e, true);
            }
        }
        for (int i = threadIdx.x; i < n * cols; i += blockDim.x) {
            const int tt = i / cols, e = i - tt * cols;
            const bool in = col0 + e < dv;
            cp_async_f32(v_s + i, vv + ((size_t)(start + c0 + tt) * heads + head) * dv + (in ? col0 + e : 0), in);
        }
        if (beta != nullptr)
            for (int i = threadIdx.x; i < n; i += blockDim.x)
                cp_async_f32(b_s + i, beta + (size_t)(start + c0 + i) * heads + head, true);
        if (MODE == kScanMemory || MODE == kScanHeadDecay)
            for (int i = threadIdx.x; i < n; i += blockDim.x)
                cp_async_f32(f_s + i, fgate + (size_t)(start + c0 + i) * heads + head, true);
        asm volatile("cp.async.commit_group;\n" ::);
    };

    issue(0, 0);
    // in the request's state the element (row r * per + il, column j) lies at [il][j][r]: a warp reads whole lines
    float* st_ptr = state + (long long)slot * state_stride + (size_t)head * per * dv * R;
    float2 S2[NC][PER / 2];                           // rows il = 2 p and 2 p + 1 of this lane
    float* top_ptr = state + (long long)slot * state_stride + aux_off + (size_t)head * dv + j;
    float top[NC];                                    // running maximum of the gates' logarithms
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        const bool live = j + c < dv;
#pragma unroll
        for (int il = 0; il < PER; il += 2) {
            S2[c][il >> 1].x = (live && il < per) ? st_ptr[((size_t)il * dv + j + c) * R + r] : 0.0f;
            S2[c][il >> 1].y = (live && il + 1 < per) ? st_ptr[((size_t)(il + 1) * dv + j + c) * R + r] : 0.0f;
        }
        top[c] = (MODE == kScanMemory && live) ? top_ptr[c] : 0.0f;
    }
    const bool has_beta = beta != nullptr;
    const float fixed = MODE == kScanFixedDecay ? fgate[head] : 1.0f;
    int stage = 0;
    for (int c0 = 0; c0 < len; c0 += kScanChunk, stage ^= 1) {
        const int n = min(kScanChunk, len - c0);
        if (c0 + kScanChunk < len) {
            issue(c0 + kScanChunk, stage ^ 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const float* k_s = sm + stage * stage_floats;
        const float* q_s = k_s + kScanChunk * L::kRow;
        const float* g_s = q_s + kScanChunk * L::kRow;
        const float* e_s = g_s + kScanChunk * L::kRow;
        const float* v_s = e_s + (MODE == kScanErase ? kScanChunk * L::kRow : 0);
        const float* b_s = v_s + kScanChunk * cols;
        const float* f_s = b_s + kScanChunk;
        // every thread walks the tokens (the shuffles want whole warps); one without a column carries zeros
        // two rows at a time with the packed float32 instructions of sm_100 (each half rounds as the scalar
        // instruction would): Sg = S g, dot += Sg k, S = Sg + k u, o += S q: four instructions for two rows
        auto step = [&](int tt, float (&o)[NC]) {
            const float4* kr = reinterpret_cast<const float4*>(k_s + tt * L::kRow + r * kLane);
            const float4* qr = reinterpret_cast<const float4*>(q_s + tt * L::kRow + r * kLane);
            const float4* gr = reinterpret_cast<const float4*>(g_s + tt * L::kRow + r * kLane);
            const float4* er = reinterpret_cast<const float4*>(e_s + tt * L::kRow + r * kLane);
            float2 kk[PER / 2];
            float2 dot_a[NC], dot_b[NC], keep2[NC];
            float write[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                dot_a[c] = dot_b[c] = make_float2(0.0f, 0.0f);
                write[c] = 1.0f;
                keep2[c] = make_float2(1.0f, 1.0f);
                if (MODE == kScanMemory) {
                    const float fi = f_s[tt], ii = b_s[tt];
                    const float top_new = fmaxf(fi + top[c], ii);
                    const float keep = expf(fi + top[c] - top_new);
                    write[c] = expf(ii - top_new);
                    top[c] = top_new;
                    keep2[c] = make_float2(keep, keep);
                } else if (MODE == kScanPlain) {
                    write[c] = has_beta ? b_s[tt] : 1.0f;
                } else if (MODE == kScanHeadDecay) {
                    keep2[c] = make_float2(b_s[tt], b_s[tt]);
                    write[c] = f_s[tt];
                } else if (MODE == kScanFixedDecay) {
                    keep2[c] = make_float2(fixed, fixed);
                }
            }
#pragma unroll
            for (int il = 0; il < PER; il += 4) {
                const float4 k4 = kr[il >> 2];
                kk[il >> 1] = make_float2(k4.x, k4.y);
                kk[(il >> 1) + 1] = make_float2(k4.z, k4.w);
                float4 g4 = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
                if (kDecayRows) g4 = gr[il >> 2];
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    float2& s0 = S2[c][il >> 1];
                    float2& s1 = S2[c][(il >> 1) + 1];
                    if (MODE == kScanErase) {                 // the removal reads the state before its decay
                        dot_a[c] = __ffma2_rn(s0, kk[il >> 1], dot_a[c]);
                        dot_b[c] = __ffma2_rn(s1, kk[(il >> 1) + 1], dot_b[c]);
                    }
                    s0 = __fmul2_rn(s0, kDecayRows ? make_float2(g4.x, g4.y) : keep2[c]);
                    s1 = __fmul2_rn(s1, kDecayRows ? make_float2(g4.z, g4.w) : keep2[c]);
                    if (MODE == kScanDelta) {
                        dot_a[c] = __ffma2_rn(s0, kk[il >> 1], dot_a[c]);
                        dot_b[c] = __ffma2_rn(s1, kk[(il >> 1) + 1], dot_b[c]);
                    }
                }
            }
            float2 u2[NC], gone[NC], o_a[NC], o_b[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float u;
                if (MODE == kScanErase) {
                    const float2 dsum = __fadd2_rn(dot_a[c], dot_b[c]);
                    const float dot = -lanes_sum<R>(dsum.x + dsum.y);
                    gone[c] = make_float2(dot, dot);
                    u = v_s[tt * cols + jl + c];
                } else if (MODE == kScanDelta) {
                    const float2 dsum = __fadd2_rn(dot_a[c], dot_b[c]);
                    const float dot = lanes_sum<R>(dsum.x + dsum.y);
                    u = b_s[tt] * (v_s[tt * cols + jl + c] - dot);
                } else {
                    u = write[c] * v_s[tt * cols + jl + c];
                }
                u2[c] = make_float2(u, u);
                o_a[c] = o_b[c] = make_float2(0.0f, 0.0f);
            }
#pragma unroll
            for (int il = 0; il < PER; il += 4) {
                const float4 q4 = qr[il >> 2];
                float4 e4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (MODE == kScanErase) e4 = er[il >> 2];
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    float2& s0 = S2[c][il >> 1];
                    float2& s1 = S2[c][(il >> 1) + 1];
                    if (MODE == kScanErase) {
                        s0 = __ffma2_rn(make_float2(e4.x, e4.y), gone[c], s0);
                        s1 = __ffma2_rn(make_float2(e4.z, e4.w), gone[c], s1);
                    }
                    s0 = __ffma2_rn(kk[il >> 1], u2[c], s0);
                    s1 = __ffma2_rn(kk[(il >> 1) + 1], u2[c], s1);
                    o_a[c] = __ffma2_rn(s0, make_float2(q4.x, q4.y), o_a[c]);
                    o_b[c] = __ffma2_rn(s1, make_float2(q4.z, q4.w), o_b[c]);
                }
            }
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float2 osum = __fadd2_rn(o_a[c], o_b[c]);
                o[c] = lanes_sum<R>(osum.x + osum.y);
                if (MODE == kScanMemory && j + c == dv - 1) o[c] = fmaxf(fabsf(o[c]), expf(-top[c])) + floor_eps;
            }
        };
        if (n == kScanChunk) {
            // a whole chunk: unrolled, the read-outs kept in registers until the end, so that no store to shared
            // memory stands between a token's loads and the next one's and they can be issued ahead
            float o_reg[kScanChunk][NC];
#pragma unroll
            for (int tt = 0; tt < kScanChunk; ++tt) step(tt, o_reg[tt]);
            if (r == 0) {
#pragma unroll
                for (int tt = 0; tt < kScanChunk; ++tt)
#pragma unroll
                    for (int c = 0; c < NC; ++c) o_s[tt * cols + jl + c] = o_reg[tt][c];
            }
        } else {
            for (int tt = 0; tt < n; ++tt) {
                float oq[NC];
                step(tt, oq);
                if (r == 0)
#pragma unroll
                    for (int c = 0; c < NC; ++c) o_s[tt * cols + jl + c] = oq[c];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < n * cols; i += blockDim.x) {
            const int tt = i / cols, e = i - tt * cols;
            const size_t at = (size_t)(start + c0 + tt) * heads + head;
            if (MODE == kScanMemory) {
                if (col0 + e < dv - 1) o_raw[at * (dv - 1) + col0 + e] = o_s[i];
                else if (col0 + e == dv - 1) den[at] = o_s[i];
            } else if (col0 + e < dv) {
                o_raw[at * dv + col0 + e] = o_s[i];
            }
        }
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        if (j + c >= dv) continue;
        if (MODE == kScanMemory && r == 0) top_ptr[c] = top[c];
#pragma unroll
        for (int il = 0; il < PER; il += 2) {
            if (il < per) st_ptr[((size_t)il * dv + j + c) * R + r] = S2[c][il >> 1].x;
            if (il + 1 < per) st_ptr[((size_t)(il + 1) * dv + j + c) * R + r] = S2[c][il >> 1].y;
        }
    }
}

// ---------------------------------------------------------------- finish
// gate_act: 0 sigmoid(gate), 1 SiLU(gate).  weight_stride: 0 where the heads share one weight of dv numbers, dv
// where every head has its own.  den: a divisor per (token, head) applied before the root mean square, or null.
__device__ __forceinline__ float finish_gate(float g, int act) {
    const float sg = 1.0f / (1.0f + expf(-g));
    return act == 1 ? g * sg : sg;
}

template <typename T, typename TG>
__global__ void delta_finish_kernel(const float* o_raw, const TG* gate, int ldg, const float* __restrict__ weight,
                                    float eps, const int* __restrict__ token_slot, int n_rows, int heads, int dv,
                                    T* out, const T* proj, int ld, int channels, int taps, float* state,
                                    long long state_stride, long long tail_off, const float* den, int gate_act,
                                    int weight_stride) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    if (slot < 0) {
        for (int e = threadIdx.x; e < heads * dv; e += blockDim.x) out[(size_t)t * heads * dv + e] = from_f32<T>(0.0f);
        return;
    }
    for (int h = warp; h < heads; h += warps) {
        const float* src = o_raw + ((size_t)t * heads + h) * dv;
        const float dn = den != nullptr ? den[(size_t)t * heads + h] : 1.0f;
        float sum = 0.0f;
        for (int e = lane; e < dv; e += 32) { const float x = src[e] / dn; sum += x * x; }
        sum = warp_sum(sum);
        const float sc = 1.0f / sqrtf(sum / (float)dv + eps);
        for (int e = lane; e < dv; e += 32) {
            const float g = to_f32<TG>(gate[(size_t)t * ldg + (size_t)h * dv + e]);
            out[((size_t)t * heads + h) * dv + e] =
                from_f32<T>(src[e] / dn * sc * weight[(size_t)h * weight_stride + e] * finish_gate(g, gate_act));
        }
    }
    // the portion's last row moves the convolution's window on: its taps - 1 newest inputs
    if (taps > 1 && (t + 1 >= n_rows || token_slot[t + 1] != slot)) {
        int len = 1;                                 // rows of the portion, as far as the window reaches
        while (len < taps - 1 && t - len >= 0 && token_slot[t - len] == slot) ++len;
        float* tail = state + (long long)slot * state_stride + tail_off;
        const int keep = taps - 1;
        for (int c = threadIdx.x; c < channels; c += blockDim.x) {
            for (int i = 0; i < keep; ++i) {         // ascending: an old entry is read before its place is written
                const int from_end = keep - i;       // this entry is the from_end-th newest input
                float x;
                if (from_end <= len) x = to_f32<T>(proj[(size_t)(t + 1 - from_end) * ld + c]);
                else x = tail[(size_t)(i + len) * channels + c];
                tail[(size_t)i * channels + c] = x;
            }
        }
    }
}

// The same with four elements per lane and access, and the window of the convolution moved eight channels at a
// time (dv a multiple of four, channels and the rows of proj multiples of eight, 16-byte boundaries).
template <typename TG> __device__ __forceinline__ float4 load_gate4(const TG* p);
template <> __device__ __forceinline__ float4 load_gate4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load_gate4<bf16>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

template <typename T, typename TG>
__global__ void delta_finish_vec_kernel(const float* o_raw, const TG* gate, int ldg, const float* __restrict__ weight,
                                        float eps, const int* __restrict__ token_slot, int n_rows, int heads, int dv,
                                        T* out, const T* proj, int ld, int channels, int taps, float* state,
                                        long long state_stride, long long tail_off, const float* den, int gate_act,
                                        int weight_stride) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    if (slot < 0) {
        for (int e = threadIdx.x; e < heads * dv; e += blockDim.x) out[(size_t)t * heads * dv + e] = from_f32<T>(0.0f);
        return;
    }
    const int Y = gridDim.y, yb = blockIdx.y;          // with few rows a token's heads and channels are dealt to gridDim.y blocks
    for (int h = heads * yb / Y + warp; h < heads * (yb + 1) / Y; h += warps) {
        const float* src = o_raw + ((size_t)t * heads + h) * dv;
        const float dn = den != nullptr ? den[(size_t)t * heads + h] : 1.0f;
        float sum = 0.0f;
        for (int e = lane * 4; e < dv; e += 128) {
            float4 v = *reinterpret_cast<const float4*>(src + e);
            v.x /= dn; v.y /= dn; v.z /= dn; v.w /= dn;
            sum += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        sum = warp_sum(sum);
        const float sc = 1.0f / sqrtf(sum / (float)dv + eps);
        for (int e = lane * 4; e < dv; e += 128) {
            const float4 v = *reinterpret_cast<const float4*>(src + e);
            const float4 g = load_gate4<TG>(gate + (size_t)t * ldg + (size_t)h * dv + e);
            const float4 w = *reinterpret_cast<const float4*>(weight + (size_t)h * weight_stride + e);
            T* dst = out + ((size_t)t * heads + h) * dv + e;
            dst[0] = from_f32<T>(v.x / dn * sc * w.x * finish_gate(g.x, gate_act));
            dst[1] = from_f32<T>(v.y / dn * sc * w.y * finish_gate(g.y, gate_act));
            dst[2] = from_f32<T>(v.z / dn * sc * w.z * finish_gate(g.z, gate_act));
            dst[3] = from_f32<T>(v.w / dn * sc * w.w * finish_gate(g.w, gate_act));
        }
    }
    if (taps > 1 && (t + 1 >= n_rows || token_slot[t + 1] != slot)) {
        int len = 1;
        while (len < taps - 1 && t - len >= 0 && token_slot[t - len] == slot) ++len;
        float* tail = state + (long long)slot * state_stride + tail_off;
        const int keep = taps - 1;
        const int cc = channels / 8;
        for (int c = (cc * yb / Y) * 8 + threadIdx.x * 8; c < (cc * (yb + 1) / Y) * 8; c += blockDim.x * 8) {
            for (int i = 0; i < keep; ++i) {         // ascending: an old entry is read before its place is written
                const int from_end = keep - i;
                float x[8];
                if (from_end <= len) Ld8<T>::load(proj + (size_t)(t + 1 - from_end) * ld + c, x);
                else Ld8<float>::load(tail + (size_t)(i + len) * channels + c, x);
                Ld8<float>::store(tail + (size_t)i * channels + c, x);
            }
        }
    }
}

// ---------------------------------------------------------------- inputs of the recurrences without a correction
// One block per token.  proj[t] = q (heads x dk) | k (heads x dk) | v (heads x dv) | anything, in the storage type;
// q times a scale, k and v as they are, all widened to float32 for the scan.  `kind` says what the gates are made of:
//   kLinearChannelDecay  z [T, heads * dk] float32 + bias: a decay per key channel, sigmoid(z)^(inv_tau), made as
//                        exp(inv_tau * logsigmoid(z));
//   kLinearLogGates      z [T, 2 heads] float32 + bias = write logits | keep logits, each capped as cap tanh(. / cap);
//                        the write's logarithm is the capped logit, the keep's is logsigmoid of its capped logit; the
//                        values get one more column of ones (the normaliser of a matrix memory), vv is [T, heads, dv + 1];
//   kLinearFixedDecay    no gates: the decays are the heads' own constants, which the scan reads itself.
// act: 0 q, k and v as projected, 1 SiLU of each (in float32, before q's scale).
enum LinearKind : int { kLinearChannelDecay = 0, kLinearLogGates = 1, kLinearFixedDecay = 2 };

__device__ __forceinline__ float linear_input(float x, int act) { return act == 1 ? x / (1.0f + expf(-x)) : x; }

__device__ __forceinline__ float log_sigmoid_f32(float z) {
    return fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
}

template <typename T>
__global__ void linear_prepare_kernel(const T* proj, int ld, const float* z, int ldz, const float* __restrict__ z_bias,
                                      int kind, int act, float p0, const int* __restrict__ token_slot, int heads, int dk, int dv,
                                      float q_scale, float* qn, float* kn, float* vv, float* decay, float* wgate,
                                      float* fgate) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    if (token_slot[t] < 0) return;
    const T* row = proj + (size_t)t * ld;
    const int qk = heads * dk;
    for (int e = threadIdx.x; e < qk; e += blockDim.x) {
        qn[(size_t)t * qk + e] = linear_input(to_f32<T>(row[e]), act) * q_scale;
        kn[(size_t)t * qk + e] = linear_input(to_f32<T>(row[qk + e]), act);
    }
    if (kind != kLinearLogGates) {
        for (int e = threadIdx.x; e < heads * dv; e += blockDim.x)
            vv[(size_t)t * heads * dv + e] = linear_input(to_f32<T>(row[2 * qk + e]), act);
    }
    if (kind == kLinearChannelDecay) {
        for (int e = threadIdx.x; e < qk; e += blockDim.x)
            decay[(size_t)t * qk + e] = expf(p0 * log_sigmoid_f32(z[(size_t)t * ldz + e] + z_bias[e]));
    } else if (kind == kLinearLogGates) {
        const int cols = dv + 1;
        for (int e = threadIdx.x; e < heads * cols; e += blockDim.x) {
            const int h = e / cols, c = e - h * cols;
            vv[(size_t)t * heads * cols + e] = c < dv ? linear_input(to_f32<T>(row[2 * qk + h * dv + c]), act) : 1.0f;
        }
        for (int h = threadIdx.x; h < heads; h += blockDim.x) {
            const float zi = z[(size_t)t * ldz + h] + z_bias[h];
            const float zf = z[(size_t)t * ldz + heads + h] + z_bias[heads + h];
            wgate[(size_t)t * heads + h] = p0 * tanhf(zi / p0);
            fgate[(size_t)t * heads + h] = log_sigmoid_f32(p0 * tanhf(zf / p0));
        }
    }
}

// kLinearFixedDecay with eight elements per access (every head's width a multiple of eight, everything on 16-byte
// boundaries): a token's q | k | v is one run of pieces, dealt to gridDim.y blocks.
template <typename T>
__global__ void linear_prepare_vec_kernel(const T* proj, int ld, int act, const int* __restrict__ token_slot, int qk, int vd,
                                          float q_scale, float* qn, float* kn, float* vv) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    if (token_slot[t] < 0) return;
    const T* row = proj + (size_t)t * ld;
    const int total = 2 * qk + vd;
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8; c < total; c += gridDim.y * blockDim.x * 8) {
        float v[8];
        Ld8<T>::load(row + c, v);
        const float scale = c < qk ? q_scale : 1.0f;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = linear_input(v[e], act) * scale;
        float* dst = c < qk ? qn + (size_t)t * qk + c : c < 2 * qk ? kn + (size_t)t * qk + (c - qk) : vv + (size_t)t * vd + (c - 2 * qk);
        Ld8<float>::store(dst, v);
    }
}

// ---------------------------------------------------------------- a read-out normed over all heads together
// out = o / sqrt(mean(o^2) + eps) * weight * act(gate), the mean over a token's `width` = heads * dv numbers.  One
// block per token; VEC: four elements per access (width and the gate's rows multiples of four, aligned).
template <typename T, typename TG, bool VEC>
__global__ void whole_finish_kernel(const float* o_raw, const TG* gate, int ldg, const float* __restrict__ weight, float eps,
                                    const int* __restrict__ token_slot, int width, T* out, int gate_act) {
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    T* dst = out + (size_t)t * width;
    if (token_slot[t] < 0) {
        for (int e = threadIdx.x; e < width; e += blockDim.x) dst[e] = from_f32<T>(0.0f);
        return;
    }
    const float* src = o_raw + (size_t)t * width;
    const TG* g = gate + (size_t)t * ldg;
    float sum = 0.0f;
    if (VEC) {
        for (int e = threadIdx.x * 4; e < width; e += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + e);
            sum += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int e = threadIdx.x; e < width; e += blockDim.x) sum += src[e] * src[e];
    }
    const float sc = 1.0f / sqrtf(block_sum(sum, scratch) / (float)width + eps);
    if (VEC) {
        for (int e = threadIdx.x * 4; e < width; e += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + e);
            const float4 x = load_gate4<TG>(g + e);
            const float4 w = *reinterpret_cast<const float4*>(weight + e);
            dst[e] = from_f32<T>(v.x * sc * w.x * finish_gate(x.x, gate_act));
            dst[e + 1] = from_f32<T>(v.y * sc * w.y * finish_gate(x.y, gate_act));
            dst[e + 2] = from_f32<T>(v.z * sc * w.z * finish_gate(x.z, gate_act));
            dst[e + 3] = from_f32<T>(v.w * sc * w.w * finish_gate(x.w, gate_act));
        }
    } else {
        for (int e = threadIdx.x; e < width; e += blockDim.x)
            dst[e] = from_f32<T>(src[e] * sc * weight[e] * finish_gate(to_f32<TG>(g[e]), gate_act));
    }
}

// ---------------------------------------------------------------- inputs of the delta rule with a removal rate per channel
// proj[t] = r | k | v | gate | a in the storage type (heads x dk, heads x dk, heads x dv, heads x dv, heads x dk), z
// [T, heads * dk] float32 the decay's logits.  Per head, with n = sqrt(sum(k^2) + unit_eps):
//   qn = r,  kn = k / n,  vv = v n  (so that kn vv^T = k v^T),  decay = exp(-rate sigmoid(z + z_bias)),
//   erase = sigmoid(a + a_bias) kn.
// One warp per head and token, all float32.
template <typename T>
__global__ void erase_prepare_kernel(const T* proj, int ld, int a_col, const float* z, int ldz, const float* __restrict__ z_bias,
                                     const float* __restrict__ a_bias, float rate, const int* __restrict__ token_slot,
                                     int heads, int dk, int dv, float unit_eps, float* qn, float* kn, float* vv, float* decay,
                                     float* erase) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    if (token_slot[t] < 0) return;
    const T* row = proj + (size_t)t * ld;
    const int qk = heads * dk, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int h = blockIdx.y * warps + (threadIdx.x >> 5); h < heads; h += gridDim.y * warps) {
        const T* k = row + qk + (size_t)h * dk;
        float sum = 0.0f;
        for (int e = lane; e < dk; e += 32) { const float x = to_f32<T>(k[e]); sum += x * x; }
        const float n = sqrtf(warp_sum(sum) + unit_eps), inv = 1.0f / n;
        for (int e = lane; e < dk; e += 32) {
            const int c = h * dk + e;
            const size_t at = (size_t)t * qk + c;
            const float u = to_f32<T>(k[e]) * inv;
            qn[at] = to_f32<T>(row[c]);
            kn[at] = u;
            decay[at] = expf(-rate / (1.0f + expf(-(z[(size_t)t * ldz + c] + z_bias[c]))));
            erase[at] = u / (1.0f + expf(-(to_f32<T>(row[a_col + c]) + a_bias[c])));
        }
        for (int e = lane; e < dv; e += 32) vv[((size_t)t * heads + h) * dv + e] = to_f32<T>(row[2 * qk + h * dv + e]) * n;
    }
}

// The same with eight elements per lane and access: a group of GS lanes (a power of two, dk <= 8 GS) holds a head, so a
// warp takes 32 / GS heads at once (dk and dv multiples of eight, everything on 16-byte boundaries).
template <typename T, int GS>
__global__ void erase_prepare_vec_kernel(const T* proj, int ld, int a_col, const float* z, int ldz, const float* __restrict__ z_bias,
                                         const float* __restrict__ a_bias, float rate, const int* __restrict__ token_slot,
                                         int heads, int dk, int dv, float unit_eps, float* qn, float* kn, float* vv,
                                         float* decay, float* erase) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    if (token_slot[t] < 0) return;
    constexpr int kPerWarp = 32 / GS;
    const T* row = proj + (size_t)t * ld;
    const int qk = heads * dk, lane = threadIdx.x & 31, grp = lane / GS, e0 = (lane % GS) * 8;
    const int per_block = (blockDim.x >> 5) * kPerWarp;
    for (int base = blockIdx.y * per_block + (threadIdx.x >> 5) * kPerWarp; base < heads; base += gridDim.y * per_block) {
        const int h = base + grp;                                   // every lane takes part in the exchange
        const bool live = h < heads && e0 < dk;
        const int c = h * dk + e0;
        const size_t at = (size_t)t * qk + c;
        float k[8] = {0, 0, 0, 0, 0, 0, 0, 0}, r[8], a[8], zz[8], zb[8], ab[8];
        if (live) {
            Ld8<T>::load(row + qk + c, k);
            Ld8<T>::load(row + c, r);
            Ld8<T>::load(row + a_col + c, a);
            Ld8<float>::load(z + (size_t)t * ldz + c, zz);
            Ld8<float>::load(z_bias + c, zb);
            Ld8<float>::load(a_bias + c, ab);
        }
        float sum = 0.0f;
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += k[e] * k[e];
#pragma unroll
        for (int o = GS / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        const float n = sqrtf(sum + unit_eps), inv = 1.0f / n;
        if (live) {
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                k[e] *= inv;
                zz[e] = expf(-rate / (1.0f + expf(-(zz[e] + zb[e]))));
                a[e] = k[e] / (1.0f + expf(-(a[e] + ab[e])));
            }
            Ld8<float>::store(qn + at, r);
            Ld8<float>::store(kn + at, k);
            Ld8<float>::store(decay + at, zz);
            Ld8<float>::store(erase + at, a);
        }
        if (h < heads)
            for (int e = e0; e < dv; e += GS * 8) {
                float v[8];
                Ld8<T>::load(row + 2 * qk + h * dv + e, v);
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] *= n;
                Ld8<float>::store(vv + ((size_t)t * heads + h) * dv + e, v);
            }
    }
}

}  // namespace tllm

using namespace tllm;

extern "C" {

// Inputs of a recurrence without a correction from the fused projections; see linear_prepare_kernel.  p0: 1 / tau
// of the channel decays, or the cap of the gates' logits.
int tllm_linear_prepare(const void* proj, int ld, int dtype, const float* z, int ldz, const float* z_bias, int kind, int act,
                        float p0, const int* token_slot, int heads, int dk, int dv, float q_scale, float* qn, float* kn,
                        float* vv, float* decay, float* wgate, float* fgate, int n_rows, cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && heads > 0 && dk > 0 && dv > 0 && p0 > 0.0f, "linear_prepare: bad sizes");
    TLLM_REQUIRE(kind == kLinearChannelDecay || kind == kLinearLogGates || kind == kLinearFixedDecay, "linear_prepare: unknown kind %d", kind);
    TLLM_REQUIRE(act == 0 || act == 1, "linear_prepare: unknown activation %d", act);
    TLLM_REQUIRE(ld >= 2 * heads * dk + heads * dv && ldz >= (kind == kLinearChannelDecay ? heads * dk : kind == kLinearLogGates ? 2 * heads : 0),
                 "linear_prepare: rows too short");
    TLLM_REQUIRE(kind == kLinearChannelDecay ? decay != nullptr : kind == kLinearFixedDecay || (wgate != nullptr && fgate != nullptr),
                 "linear_prepare: no place for the gates");
    if (n_rows == 0) return 0;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    if (kind == kLinearFixedDecay && (heads * dk) % 8 == 0 && (heads * dv) % 8 == 0 && ld % 8 == 0 && al(proj) && al(qn) && al(kn) && al(vv)) {
        const int qk = heads * dk, vd = heads * dv, pieces = (2 * qk + vd) / 8;
        const int sms = sm_count_cached() > 0 ? sm_count_cached() : 148;
        int split = 1;                                  // blocks per token where few rows leave the GPU empty
        while (split * 2 * 128 <= pieces && (long long)n_rows * split < 2LL * sms) split *= 2;
        const dim3 grid(n_rows, split), block(128);
        if (dtype == kBF16)
            launch_pdl(kPdlOther, linear_prepare_vec_kernel<bf16>, grid, block, 0, stream, (const bf16*)proj, ld, act, token_slot, qk, vd, q_scale, qn, kn, vv);
        else if (dtype == kF32)
            launch_pdl(kPdlOther, linear_prepare_vec_kernel<float>, grid, block, 0, stream, (const float*)proj, ld, act, token_slot, qk, vd, q_scale, qn, kn, vv);
        else TLLM_REQUIRE(false, "linear_prepare: unknown dtype %d", dtype);
        return finish_launch("linear_prepare");
    }
    if (dtype == kBF16)
        launch_pdl(kPdlOther, linear_prepare_kernel<bf16>, dim3(n_rows), dim3(256), 0, stream, (const bf16*)proj, ld, z, ldz,
                   z_bias, kind, act, p0, token_slot, heads, dk, dv, q_scale, qn, kn, vv, decay, wgate, fgate);
    else if (dtype == kF32)
        launch_pdl(kPdlOther, linear_prepare_kernel<float>, dim3(n_rows), dim3(256), 0, stream, (const float*)proj, ld, z, ldz,
                   z_bias, kind, act, p0, token_slot, heads, dk, dv, q_scale, qn, kn, vv, decay, wgate, fgate);
    else TLLM_REQUIRE(false, "linear_prepare: unknown dtype %d", dtype);
    return finish_launch("linear_prepare");
}

// See erase_prepare_kernel.  a_col: column of the removal rates' logits in a row of proj.
int tllm_erase_prepare(const void* proj, int ld, int dtype, int a_col, const float* z, int ldz, const float* z_bias,
                       const float* a_bias, float rate, const int* token_slot, int heads, int dk, int dv, float unit_eps,
                       float* qn, float* kn, float* vv, float* decay, float* erase, int n_rows, cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && heads > 0 && dk > 0 && dv > 0 && unit_eps > 0.0f, "erase_prepare: bad sizes");
    TLLM_REQUIRE(a_col >= heads * (2 * dk + dv) && ld >= a_col + heads * dk && ldz >= heads * dk, "erase_prepare: rows too short");
    TLLM_REQUIRE(dtype == kBF16 || dtype == kF32, "erase_prepare: unknown dtype %d", dtype);
    if (n_rows == 0) return 0;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const bool vec = dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && ld % 8 == 0 && a_col % 8 == 0 && ldz % 4 == 0 && al(proj) && al(z) &&
                     al(z_bias) && al(a_bias) && al(qn) && al(kn) && al(vv) && al(decay) && al(erase);
    int gs = 1;
    while (gs * 8 < dk) gs *= 2;
    const int per_warp = vec ? 32 / gs : 1;
    // blocks per token: a warp's heads each where few rows leave the GPU empty
    const int sms = sm_count_cached() > 0 ? sm_count_cached() : 148;
    int warps = 8, split = 1;
    while (warps > 1 && (warps / 2) * per_warp >= heads) warps /= 2;
    while (split * warps * per_warp < heads && (long long)n_rows * split < 2LL * sms) split *= 2;
    while (warps > 2 && split * 2 <= 64 && (long long)n_rows * split * 2 <= 2LL * sms) { warps /= 2; split *= 2; }
    const dim3 grid(n_rows, split), block(warps * 32);
#define EP(T) launch_pdl(kPdlOther, erase_prepare_kernel<T>, grid, block, 0, stream, (const T*)proj, ld, a_col, z, ldz, z_bias, a_bias, \
                         rate, token_slot, heads, dk, dv, unit_eps, qn, kn, vv, decay, erase)
#define EPV(T, G) launch_pdl(kPdlOther, erase_prepare_vec_kernel<T, G>, grid, block, 0, stream, (const T*)proj, ld, a_col, z, ldz, z_bias, \
                             a_bias, rate, token_slot, heads, dk, dv, unit_eps, qn, kn, vv, decay, erase)
#define EPG(T)                             \
    do {                                   \
        if (!vec) EP(T);                   \
        else if (gs == 1) EPV(T, 1);       \
        else if (gs == 2) EPV(T, 2);       \
        else if (gs == 4) EPV(T, 4);       \
        else if (gs == 8) EPV(T, 8);       \
        else if (gs == 16) EPV(T, 16);     \
        else EPV(T, 32);                   \
    } while (0)
    if (dtype == kBF16) EPG(bf16);
    else EPG(float);
#undef EPG
#undef EPV
#undef EP
    return finish_launch("erase_prepare");
}

// Lanes that share a column of the state for keys of width dk (the state's layout depends on it).
int tllm_delta_rule_lanes(int dk) { return delta_lanes(dk); }

// Floats of one request's state: S of every head in the scan's layout, then the convolution's window.
long long tllm_delta_rule_state_floats(int heads, int kv_heads, int dk, int dv, int taps) {
    const int r = delta_lanes(dk), per = (dk + r - 1) / r;
    return (long long)heads * per * r * dv + (long long)(taps - 1) * (2 * kv_heads * dk + heads * dv);
}

// conv_w [channels, taps], and conv_t, the same taps as [taps, channels] (null: the scalar kernel serves).
int tllm_delta_prepare(const void* proj, int ld, int dtype, const void* conv_w, const void* conv_t, int taps, const float* a,
                       int lda, const float* dt_bias, const float* rate, const int* token_slot, const float* state,
                       long long state_stride, int heads, int kv_heads, int dk, int dv, float q_scale,
                       float unit_eps, float* qn, float* kn, float* vv, float* decay, float* beta, int n_rows,
                       int decay_per_head, int beta_col, cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dv > 0 && taps > 0,
                 "delta_prepare: bad sizes");
    const int channels = 2 * kv_heads * dk + heads * dv;
    if (beta_col < 0) beta_col = channels;
    TLLM_REQUIRE(ld >= beta_col + heads && beta_col >= channels && lda >= (decay_per_head ? heads : heads * dk),
                 "delta_prepare: rows too short");
    if (n_rows == 0) return 0;
    const int r = delta_lanes(dk), per = (dk + r - 1) / r;
    TLLM_REQUIRE(per <= kScanMaxPer, "delta_prepare: keys of width %d are too wide", dk);
    const long long tail_off = (long long)heads * per * r * dv;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const bool vec = conv_t != nullptr && dk % 8 == 0 && dv % 8 == 0 && ld % 8 == 0 && tail_off % 4 == 0 &&
                     (decay_per_head || (lda % 4 == 0 && al(a) && al(dt_bias))) &&
                     state_stride % 4 == 0 && al(proj) && al(conv_t) && al(state) && al(qn) && al(kn) &&
                     al(vv) && al(decay);
    // blocks per token: one where the rows fill the GPU, else up to a q or k head each
    const int sms_p = sm_count_cached() > 0 ? sm_count_cached() : 148;
    int split = 1;
    if (vec) while (split * 2 <= 2 * kv_heads && (long long)n_rows * split < 2LL * sms_p) split *= 2;
    const size_t smem = (size_t)(vec ? (2 * kv_heads + split - 1) / split * dk + dk : channels) * sizeof(float);
    TLLM_REQUIRE(smem <= 200 * 1024, "delta_prepare: %d channels do not fit in shared memory", channels);
#define PREP_VEC(T, N)                                                                                           \
    do {                                                                                                         \
        if (smem > 48 * 1024) {                                                                                  \
            cudaError_t e = cudaFuncSetAttribute(delta_prepare_vec_kernel<T, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) { set_error("delta_prepare: %s", cudaGetErrorString(e)); return (int)e; }      \
        }                                                                                                        \
        launch_pdl(kPdlOther, delta_prepare_vec_kernel<T, N>, dim3(n_rows, split), dim3(split > 1 ? 128 : 256), smem, stream, \
                   (const T*)proj, ld, (const T*)conv_t, taps, a, lda, dt_bias, rate, token_slot, state, state_stride,   \
                   tail_off, heads, kv_heads, dk, dv, q_scale, unit_eps, qn, kn, vv, decay, beta, n_rows,      \
                   decay_per_head, beta_col);                                                                    \
    } while (0)
#define PREP(T)                                                                                                  \
    do {                                                                                                         \
        if (vec) {                                                                                               \
            if (taps == 2) PREP_VEC(T, 2);                                                                       \
            else if (taps == 3) PREP_VEC(T, 3);                                                                  \
            else if (taps == 4) PREP_VEC(T, 4);                                                                  \
            else PREP_VEC(T, 0);                                                                                 \
            break;                                                                                               \
        }                                                                                                        \
        if (smem > 48 * 1024) {                                                                                  \
            cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) { set_error("delta_prepare: %s", cudaGetErrorString(e)); return (int)e; }      \
        }                                                                                                        \
        launch_pdl(kPdlOther, delta_prepare_kernel<T>, dim3(n_rows), dim3(256), smem, stream, (const T*)proj, ld, \
                   (const T*)conv_w, taps, a, lda, dt_bias, rate, token_slot, state, state_stride, tail_off,     \
                   heads, kv_heads, dk, dv, q_scale, unit_eps, qn, kn, vv, decay, beta, n_rows,                  \
                   decay_per_head, beta_col);                                                                    \
    } while (0)
    if (dtype == kBF16) PREP(bf16);
    else if (dtype == kF32) PREP(float);
    else TLLM_REQUIRE(false, "delta_prepare: unknown dtype %d", dtype);
#undef PREP
#undef PREP_VEC
    return finish_launch("delta_prepare");
}

// seg_info: int[segments][4] = slot, first row, length, first position; null: every row is a portion of one token.
// rows: rows of the step (how long the portions are on average decides how many columns a thread takes).
int tllm_delta_scan(const int* seg_info, int segments, int rows, const int* token_slot, const float* qn, const float* kn,
                    const float* vv, const float* decay, const float* beta, float* state, long long state_stride,
                    int heads, int kv_heads, int dk, int dv, float* o_raw, int mode, const float* fgate,
                    const float* erase, long long aux_off, float floor_eps, float* den, cudaStream_t stream) {
    TLLM_REQUIRE(segments >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dv > 0,
                 "delta_scan: bad sizes");
    TLLM_REQUIRE(mode == kScanDelta || mode == kScanPlain || mode == kScanMemory || mode == kScanHeadDecay || mode == kScanErase ||
                 mode == kScanFixedDecay,
                 "delta_scan: unknown recurrence %d", mode);
    TLLM_REQUIRE(mode == kScanMemory ? (beta != nullptr && fgate != nullptr && den != nullptr && dv >= 2 && aux_off > 0)
                 : mode == kScanHeadDecay ? (beta != nullptr && fgate != nullptr) : mode == kScanFixedDecay ? fgate != nullptr : decay != nullptr, "delta_scan: the recurrence lacks an operand");
    TLLM_REQUIRE(mode != kScanDelta || beta != nullptr, "delta_scan: the delta rule needs its betas");
    TLLM_REQUIRE(mode != kScanErase || (erase != nullptr && kv_heads == heads), "delta_scan: a removal per channel needs its rates and a key per head");
    TLLM_REQUIRE(heads <= 65535, "delta_scan: %d heads", heads);
    if (segments == 0) return 0;
    const int r = delta_lanes(dk), per = (dk + r - 1) / r;
    TLLM_REQUIRE(per <= kScanMaxPer, "delta_scan: keys of width %d are too wide", dk);
    // columns per block: whole warps, at most 256 threads, not wider than the values, and at least a block per
    // multiprocessor in all where the value width allows it (a column does not depend on the others, so the
    // result is the same however they are dealt)
    int cols = 256 / r;
    const int sms = sm_count_cached() > 0 ? sm_count_cached() : 148;
    // two columns per thread where a multiprocessor has so many columns that reading the tokens' rows for each would take
    // longer than a column's own chain of sums (measured: 4096 columns of 128 rows gain 12 to 18%, 2048 lose 5%)
    const bool two = r < 32 && per > 8 && seg_info != nullptr && rows >= 16LL * segments && (long long)segments * heads * dv >= 24LL * sms;
    const int nc = two ? 2 : 1;
    const int min_cols = nc * (32 / r > 1 ? 32 / r : 1);
    while (cols > min_cols && cols / 2 >= dv) cols /= 2;
    while (cols > min_cols && (long long)segments * heads * ((dv + cols - 1) / cols) < (nc == 2 ? sms * 3 / 4 : sms)) cols /= 2;
    const int col_blocks = (dv + cols - 1) / cols;
    const int threads = cols / nc * r;
    TLLM_REQUIRE(col_blocks <= 65535, "delta_scan: sizes %d x %d do not fit", dk, dv);
    const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const int vec = dk % 4 == 0 && per % 4 == 0 && aligned(qn) && aligned(kn) && (decay == nullptr || aligned(decay)) &&
                    (erase == nullptr || aligned(erase));
#define SCAN(RR, PP)                                                                                             \
    do {                                                                                                         \
        if (mode == kScanDelta) SCAN_MODE(RR, PP, kScanDelta);                                                   \
        else if (mode == kScanPlain) SCAN_MODE(RR, PP, kScanPlain);                                              \
        else if (mode == kScanHeadDecay) SCAN_MODE(RR, PP, kScanHeadDecay);                                      \
        else if (mode == kScanErase) SCAN_MODE(RR, PP, kScanErase);                                              \
        else if (mode == kScanFixedDecay) SCAN_MODE(RR, PP, kScanFixedDecay);                                    \
        else SCAN_MODE(RR, PP, kScanMemory);                                                                     \
    } while (0)
#define SCAN_MODE(RR, PP, MM)                                                                                           \
    do {                                                                                                         \
        if (nc == 2) SCAN_NC(RR, PP, MM, (RR < 32 && PP == 16 ? 2 : 1));                                         \
        else SCAN_NC(RR, PP, MM, 1);                                                                             \
    } while (0)
#define SCAN_NC(RR, PP, MM, NN)                                                                                  \
    do {                                                                                                         \
        const size_t smem = ((size_t)2 * ScanLayout<RR, PP, scan_vecs(MM)>::stage_floats(cols) + (size_t)scan_chunk(RR) * cols) * sizeof(float); \
        TLLM_REQUIRE(smem <= 200 * 1024, "delta_scan: sizes %d x %d do not fit", dk, dv);                         \
        static OncePerDevice configured;                                                                         \
        if (configured.first()) {                                                                                \
            cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<RR, PP, MM, NN>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
            if (e != cudaSuccess) { set_error("delta_scan: %s", cudaGetErrorString(e)); return (int)e; }         \
            configured.done();                                                                                   \
        }                                                                                                        \
        launch_pdl(kPdlOther, delta_scan_kernel<RR, PP, MM, NN>, dim3(segments, heads, col_blocks), dim3(threads), smem, stream, \
                   seg_info, token_slot, qn, kn, vv, decay, beta, state, state_stride, heads, kv_heads, dk, dv,  \
                   cols, vec, o_raw, fgate, erase, aux_off, floor_eps, den);                                            \
    } while (0)
    if (r == 4 && per <= 4) SCAN(4, 4);
    else if (r == 4 && per <= 8) SCAN(4, 8);
    else if (r == 4) SCAN(4, 16);
    else if (r == 8) SCAN(8, 16);
    else if (r == 16) SCAN(16, 16);
    else SCAN(32, 16);
#undef SCAN
#undef SCAN_MODE
#undef SCAN_NC
    return finish_launch("delta_scan");
}

// The read-out of all heads normed together; see whole_finish_kernel.  gate: float32 (gate_f32) or the storage type.
int tllm_whole_finish(const float* o_raw, const void* gate, int gate_f32, int ldg, const float* weight, float eps,
                      const int* token_slot, int n_rows, int width, void* out, int dtype, int gate_act, cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && width > 0 && eps > 0.0f && ldg >= width, "whole_finish: bad sizes");
    TLLM_REQUIRE(gate_act == 0 || gate_act == 1, "whole_finish: bad options");
    if (n_rows == 0) return 0;
    const auto al = [](const void* p, unsigned to) { return (reinterpret_cast<uintptr_t>(p) & (to - 1)) == 0; };
    const bool vec = width % 4 == 0 && ldg % 4 == 0 && al(o_raw, 16) && al(weight, 16) && al(gate, gate_f32 || dtype == kF32 ? 16 : 8);
    int threads = 64;                                   // about two accesses of four per thread
    while (threads < 512 && threads * 8 < width) threads *= 2;
#define WHOLE(T, TG)                                                                                                        \
    do {                                                                                                                    \
        if (vec) launch_pdl(kPdlOther, whole_finish_kernel<T, TG, true>, dim3(n_rows), dim3(threads), 0, stream, o_raw,      \
                            (const TG*)gate, ldg, weight, eps, token_slot, width, (T*)out, gate_act);                       \
        else launch_pdl(kPdlOther, whole_finish_kernel<T, TG, false>, dim3(n_rows), dim3(threads), 0, stream, o_raw,         \
                        (const TG*)gate, ldg, weight, eps, token_slot, width, (T*)out, gate_act);                           \
    } while (0)
    if (dtype == kBF16) { if (gate_f32) WHOLE(bf16, float); else WHOLE(bf16, bf16); }
    else if (dtype == kF32) WHOLE(float, float);
    else TLLM_REQUIRE(false, "whole_finish: unknown dtype %d", dtype);
#undef WHOLE
    return finish_launch("whole_finish");
}

// gate: float32 (gate_f32) or the storage type; state_dv: value columns of S in the state's layout (dv, or more where
// the recurrence keeps columns of its own); with taps 1 neither proj nor the state are touched.
int tllm_delta_finish(const float* o_raw, const void* gate, int gate_f32, int ldg, const float* weight, float eps,
                      const int* token_slot, int n_rows, int heads, int kv_heads, int dk, int dv, void* out,
                      int dtype, const void* proj, int ld, int taps, float* state, long long state_stride,
                      const float* den, int gate_act, int weight_stride, cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && heads > 0 && dv > 0 && eps > 0.0f && ldg >= heads * dv, "delta_finish: bad sizes");
    TLLM_REQUIRE((gate_act == 0 || gate_act == 1) && (weight_stride == 0 || weight_stride == dv), "delta_finish: bad options");
    if (n_rows == 0) return 0;
    const int channels = 2 * kv_heads * dk + heads * dv;
    const int r = delta_lanes(dk), per = (dk + r - 1) / r;
    const long long tail_off = (long long)heads * per * r * dv;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const bool vec = dv % 4 == 0 && ldg % 4 == 0 && al(o_raw) && (reinterpret_cast<uintptr_t>(gate) & 7u) == 0 && al(weight) &&
                     (gate_f32 || dtype == kF32 ? al(gate) : true) &&
                     (taps <= 1 || (channels % 8 == 0 && ld % 8 == 0 && tail_off % 4 == 0 && state_stride % 4 == 0 && al(proj) && al(state)));
    const int sms_f = sm_count_cached() > 0 ? sm_count_cached() : 148;
    int split = 1;
    while (vec && split * 2 <= heads && (long long)n_rows * split < 2LL * sms_f) split *= 2;
#define FIN(T, TG)                                                                                                         \
    do {                                                                                                                   \
        if (vec)                                                                                                           \
            launch_pdl(kPdlOther, delta_finish_vec_kernel<T, TG>, dim3(n_rows, split), dim3(split > 1 ? 128 : 256), 0, stream, o_raw, (const TG*)gate, ldg, weight, eps, \
                       token_slot, n_rows, heads, dv, (T*)out, (const T*)proj, ld, channels, taps, state, state_stride, tail_off, den, gate_act, weight_stride); \
        else                                                                                                               \
            launch_pdl(kPdlOther, delta_finish_kernel<T, TG>, dim3(n_rows), dim3(256), 0, stream, o_raw, (const TG*)gate, ldg, weight, eps, \
                       token_slot, n_rows, heads, dv, (T*)out, (const T*)proj, ld, channels, taps, state, state_stride, tail_off, den, gate_act, weight_stride); \
    } while (0)
    if (dtype == kBF16) { if (gate_f32) FIN(bf16, float); else FIN(bf16, bf16); }
    else if (dtype == kF32) FIN(float, float);
    else TLLM_REQUIRE(false, "delta_finish: unknown dtype %d", dtype);
#undef FIN
    return finish_launch("delta_finish");
}

}  // extern "C"
