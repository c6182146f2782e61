// Several residual streams side by side ("hyper-connections"): x [T][S][width] float32.  A sub-layer reads a weighted
// sum of the streams and its output is written back to all of them, mixed:
//
//   x_t <- sum_s mix[s, t] x_s + out[t] y,     y = (delta + bias) * sigmoid(gate + gate_bias),
//   u = sum_t in[t] x_t,   h = gain * u / sqrt(mean(u^2) + eps),
//   and, for a sub-layer whose input is shifted by a token,  h + (h' - h) * shift  with h' the previous token's h.
//
// One kernel, `stream_read`, does all of it between two sub-layers: the update that the last one left (if any), the
// new streams written back, the weighted sum, its norm and the shift; delta, gate and h are in the storage type, all
// arithmetic is float32.  A block walks a run of consecutive rows and keeps the last h in registers; the row before
// its run is computed once more (not written), so that no block waits for another.  That is why the new streams go to
// a buffer of their own.  The h of the token before a portion comes from the request's state `tail` [slots][width]
// (zeros at admission).  In a step of single tokens the kernel moves that state on itself; where portions are longer,
// another block may still read it, and `stream_tails` does it afterwards.
#include "common.cuh"

namespace tllm {

template <typename T> struct Row8;
template <> struct Row8<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[8]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
};
template <> struct Row8<bf16> {
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

struct StreamArgs {
    const float* x;              // [T][S][width]
    float* x_new;                // the same after the update; null: not written
    const void* delta;           // [T][width] in the storage type; null: no update
    const float* delta_bias;     // [width] or null
    const void* gate;            // [T][width] logits in the storage type; null: no gate
    const float* gate_bias;      // [width] or null
    const float* mix;            // [S][S], from | to
    const float* out;            // [S]
    const float* in;             // [S]; null: the plain sum
    const float* gain;           // [width]
    float eps;
    void* h;                     // [rows][width] in the storage type
    const float* shift;          // [width]; null: no shift
    void* shifted;               // [T][width] in the storage type
    float* tail;                 // [slots][tail_stride]: the previous token's h per request
    long long tail_stride;
    int save_tails;              // move the tails on (steps of single tokens)
    const int* token_slot;
    const int* rows;             // rows to read (no update is written, no shift); null: all
    int n_rows, width, streams, run;
};

// CHUNKS groups of eight columns per thread (width <= blockDim * 8 * CHUNKS, a multiple of eight).
template <typename T, int S, int CHUNKS>
__global__ void __launch_bounds__(512)
stream_read_vec_kernel(const StreamArgs a) {
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int n_chunks = a.width >> 3;
    const T* delta = (const T*)a.delta;
    const T* gate = (const T*)a.gate;
    float w_in[S], w_out[S], w_mix[S][S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        w_in[s] = a.in != nullptr ? a.in[s] : 1.0f;
        w_out[s] = delta != nullptr ? a.out[s] : 0.0f;
#pragma unroll
        for (int t = 0; t < S; ++t) w_mix[s][t] = delta != nullptr ? a.mix[s * S + t] : (s == t ? 1.0f : 0.0f);
    }
    // h of one row, rounded to the storage type (what the sub-layer and the next token's shift see)
    auto row_h = [&](int r, bool write, float (&h)[CHUNKS][8]) {
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < CHUNKS; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= n_chunks) continue;
            float x[S][8], y[8], z[8];
#pragma unroll
            for (int s = 0; s < S; ++s) Row8<float>::load(a.x + ((size_t)r * S + s) * a.width + c * 8, x[s]);
            if (delta != nullptr) {
                Row8<T>::load(delta + (size_t)r * a.width + c * 8, y);
                if (gate != nullptr) Row8<T>::load(gate + (size_t)r * a.width + c * 8, z);
                if (a.delta_bias != nullptr) {
                    float b[8];
                    Row8<float>::load(a.delta_bias + c * 8, b);
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] += b[e];
                }
                if (gate != nullptr) {
                    float b[8] = {0, 0, 0, 0, 0, 0, 0, 0};
                    if (a.gate_bias != nullptr) Row8<float>::load(a.gate_bias + c * 8, b);
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] *= 1.0f / (1.0f + expf(-(z[e] + b[e])));
                }
                float nx[S][8];
#pragma unroll
                for (int t = 0; t < S; ++t)
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        float v = w_mix[0][t] * x[0][e];
#pragma unroll
                        for (int s = 1; s < S; ++s) v += w_mix[s][t] * x[s][e];
                        nx[t][e] = v + w_out[t] * y[e];
                    }
#pragma unroll
                for (int t = 0; t < S; ++t) {
#pragma unroll
                    for (int e = 0; e < 8; ++e) x[t][e] = nx[t][e];
                    if (write && a.x_new != nullptr) Row8<float>::store(a.x_new + ((size_t)r * S + t) * a.width + c * 8, x[t]);
                }
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                float u = w_in[0] * x[0][e];
#pragma unroll
                for (int s = 1; s < S; ++s) u += w_in[s] * x[s][e];
                h[j][e] = u;
                sum += u * u;
            }
        }
        sum = block_sum(sum, scratch);
        const float sc = 1.0f / sqrtf(sum / (float)a.width + a.eps);
#pragma unroll
        for (int j = 0; j < CHUNKS; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= n_chunks) continue;
            float g[8];
            Row8<float>::load(a.gain + c * 8, g);
#pragma unroll
            for (int e = 0; e < 8; ++e) h[j][e] = to_f32<T>(from_f32<T>(g[e] * h[j][e] * sc));
        }
    };
    T* h_out = (T*)a.h;
    if (a.rows != nullptr) {
        const int r = a.rows[blockIdx.x];
        float h[CHUNKS][8];
        if (r >= 0) row_h(r, false, h);
#pragma unroll
        for (int j = 0; j < CHUNKS; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= n_chunks) continue;
            if (r < 0)
#pragma unroll
                for (int e = 0; e < 8; ++e) h[j][e] = 0.0f;
            Row8<T>::store(h_out + (size_t)blockIdx.x * a.width + c * 8, h[j]);
        }
        return;
    }
    const int r0 = blockIdx.x * a.run, r1 = min(r0 + a.run, a.n_rows);
    float prev[CHUNKS][8];
    int prev_slot = -1;
    if (a.shift != nullptr && r0 > 0 && a.token_slot[r0] >= 0 && a.token_slot[r0 - 1] == a.token_slot[r0]) {
        row_h(r0 - 1, false, prev);
        prev_slot = a.token_slot[r0];
    }
    for (int r = r0; r < r1; ++r) {
        float h[CHUNKS][8];
        row_h(r, true, h);
        const int slot = a.shift != nullptr ? a.token_slot[r] : -1;
        const bool last = slot >= 0 && a.save_tails && (r + 1 >= a.n_rows || a.token_slot[r + 1] != slot);
#pragma unroll
        for (int j = 0; j < CHUNKS; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= n_chunks) continue;
            Row8<T>::store(h_out + (size_t)r * a.width + c * 8, h[j]);
            if (a.shift == nullptr) continue;
            float p[8] = {0, 0, 0, 0, 0, 0, 0, 0}, w[8];
            if (slot >= 0 && prev_slot == slot) {
#pragma unroll
                for (int e = 0; e < 8; ++e) p[e] = prev[j][e];
            } else if (slot >= 0) {
                Row8<float>::load(a.tail + (long long)slot * a.tail_stride + c * 8, p);
            }
            Row8<float>::load(a.shift + c * 8, w);
#pragma unroll
            for (int e = 0; e < 8; ++e) p[e] = h[j][e] + (p[e] - h[j][e]) * w[e];
            Row8<T>::store((T*)a.shifted + (size_t)r * a.width + c * 8, p);
            if (last) Row8<float>::store(a.tail + (long long)slot * a.tail_stride + c * 8, h[j]);
#pragma unroll
            for (int e = 0; e < 8; ++e) prev[j][e] = h[j][e];
        }
        prev_slot = slot;
    }
}

// Any width, any number of streams: a row of h and the one before it in shared memory, element by element.
template <typename T>
__global__ void stream_read_kernel(const StreamArgs a) {
    extern __shared__ float rows_smem[];            // [2][width]
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int S = a.streams, W = a.width;
    const T* delta = (const T*)a.delta;
    const T* gate = (const T*)a.gate;
    auto row_h = [&](int r, bool write, float* h) {
        float sum = 0.0f;
        for (int i = threadIdx.x; i < W; i += blockDim.x) {
            float y = 0.0f;
            if (delta != nullptr) {
                y = to_f32<T>(delta[(size_t)r * W + i]) + (a.delta_bias != nullptr ? a.delta_bias[i] : 0.0f);
                if (gate != nullptr)
                    y *= 1.0f / (1.0f + expf(-(to_f32<T>(gate[(size_t)r * W + i]) + (a.gate_bias != nullptr ? a.gate_bias[i] : 0.0f))));
            }
            float u = 0.0f;
            for (int t = 0; t < S; ++t) {
                float v;
                if (delta != nullptr) {
                    v = 0.0f;
                    for (int s = 0; s < S; ++s) v += a.mix[s * S + t] * a.x[((size_t)r * S + s) * W + i];
                    v += a.out[t] * y;
                    if (write && a.x_new != nullptr) a.x_new[((size_t)r * S + t) * W + i] = v;
                } else {
                    v = a.x[((size_t)r * S + t) * W + i];
                }
                u += (a.in != nullptr ? a.in[t] : 1.0f) * v;
            }
            h[i] = u;
            sum += u * u;
        }
        sum = block_sum(sum, scratch);
        const float sc = 1.0f / sqrtf(sum / (float)W + a.eps);
        for (int i = threadIdx.x; i < W; i += blockDim.x) h[i] = to_f32<T>(from_f32<T>(a.gain[i] * h[i] * sc));
    };
    T* h_out = (T*)a.h;
    if (a.rows != nullptr) {
        const int r = a.rows[blockIdx.x];
        if (r >= 0) row_h(r, false, rows_smem);
        for (int i = threadIdx.x; i < W; i += blockDim.x)
            h_out[(size_t)blockIdx.x * W + i] = from_f32<T>(r >= 0 ? rows_smem[i] : 0.0f);
        return;
    }
    const int r0 = blockIdx.x * a.run, r1 = min(r0 + a.run, a.n_rows);
    float* cur = rows_smem;
    float* prev = rows_smem + W;
    int prev_slot = -1;
    if (a.shift != nullptr && r0 > 0 && a.token_slot[r0] >= 0 && a.token_slot[r0 - 1] == a.token_slot[r0]) {
        row_h(r0 - 1, false, prev);
        prev_slot = a.token_slot[r0];
    }
    for (int r = r0; r < r1; ++r) {                 // a thread meets only its own elements of the two rows
        row_h(r, true, cur);
        const int slot = a.shift != nullptr ? a.token_slot[r] : -1;
        const bool last = slot >= 0 && a.save_tails && (r + 1 >= a.n_rows || a.token_slot[r + 1] != slot);
        for (int i = threadIdx.x; i < W; i += blockDim.x) {
            const float h = cur[i];
            h_out[(size_t)r * W + i] = from_f32<T>(h);
            if (a.shift == nullptr) continue;
            float p = 0.0f;
            if (slot >= 0) p = prev_slot == slot ? prev[i] : a.tail[(long long)slot * a.tail_stride + i];
            ((T*)a.shifted)[(size_t)r * W + i] = from_f32<T>(h + (p - h) * a.shift[i]);
            if (last) a.tail[(long long)slot * a.tail_stride + i] = h;
        }
        float* other = prev;
        prev = cur;
        cur = other;
        prev_slot = slot;
    }
}

// The tails of a step with portions: one block per portion copies the h of its last row.
template <typename T>
__global__ void stream_tails_kernel(const int* __restrict__ seg_info, const T* h, float* tail, long long tail_stride, int width) {
    TLLM_PDL_ENTER();
    const int slot = seg_info[4 * blockIdx.x], row = seg_info[4 * blockIdx.x + 1] + seg_info[4 * blockIdx.x + 2] - 1;
    if (slot < 0) return;
    for (int i = threadIdx.x; i < width; i += blockDim.x)
        tail[(long long)slot * tail_stride + i] = to_f32<T>(h[(size_t)row * width + i]);
}

// ---------------------------------------------------------------- embedding with sinusoids
// out[t, s, :] = table[ids[t], :] * scale + position vector, the same for every stream s: column 2 i of the position
// vector is sin(p f_i), column 2 i + 1 cos(p f_i).  A frequency comes as two floats (its rounded value and what the
// rounding left): the product p f_i is formed with its own rounding error beside it, and sine and cosine are those of
// the sum of the two (a few terms of the small one's series), so that angles of many turns keep float32 accuracy.
template <typename TW>
__global__ void embedding_sinusoid_kernel(const int* __restrict__ ids, const int* __restrict__ positions,
                                          const TW* __restrict__ table, const float2* __restrict__ freq, float scale,
                                          float* __restrict__ out, int width, int vocab, int streams) {
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    int id = ids[t];
    const bool pad = id < 0;
    if (id >= vocab) id = vocab - 1;
    const TW* src = table + (size_t)(pad ? 0 : id) * width;
    float* dst = out + (size_t)t * streams * width;
    const float p = (float)positions[t];
    for (int i = threadIdx.x; 2 * i < width; i += blockDim.x) {
        float a = 0.0f, b = 0.0f;
        const bool two = 2 * i + 1 < width;
        if (!pad) {
            const float2 f = freq[i];
            const float ang = p * f.x, rest = fmaf(p, f.y, fmaf(p, f.x, -ang));
            float sn, cs;
            sincosf(ang, &sn, &cs);
            const float c2 = 1.0f - 0.5f * rest * rest, s2 = rest * (1.0f - rest * rest * (1.0f / 6.0f));   // cos, sin of rest
            a = to_f32<TW>(src[2 * i]) * scale + fmaf(sn, c2, cs * s2);
            if (two) b = to_f32<TW>(src[2 * i + 1]) * scale + fmaf(cs, c2, -sn * s2);
        }
        for (int s = 0; s < streams; ++s) {
            dst[(size_t)s * width + 2 * i] = a;
            if (two) dst[(size_t)s * width + 2 * i + 1] = b;
        }
    }
}

}  // namespace tllm

using namespace tllm;

extern "C" {

// See StreamArgs.  rows: read only these rows' sums (the model's last norm); then nothing else is written.
int tllm_stream_read(const float* x, float* x_new, const void* delta, const float* delta_bias, const void* gate,
                     const float* gate_bias, const float* mix, const float* out, const float* in, const float* gain,
                     float eps, void* h, int dtype, const float* shift, void* shifted, float* tail, long long tail_stride,
                     int save_tails, const int* token_slot, const int* rows, int n_rows, int width, int streams,
                     cudaStream_t stream) {
    TLLM_REQUIRE(n_rows >= 0 && width > 0 && streams > 0 && eps > 0.0f, "stream_read: bad sizes");
    TLLM_REQUIRE(x != nullptr && gain != nullptr && h != nullptr && x_new != x, "stream_read: missing operand");
    TLLM_REQUIRE(delta == nullptr || (mix != nullptr && out != nullptr), "stream_read: an update without its weights");
    TLLM_REQUIRE(delta == nullptr || rows != nullptr || x_new != nullptr, "stream_read: an update with no place to go");
    TLLM_REQUIRE(shift == nullptr || (rows == nullptr && shifted && tail && token_slot), "stream_read: a shift without its operands");
    TLLM_REQUIRE(dtype == kBF16 || dtype == kF32, "stream_read: unknown dtype %d", dtype);
    if (n_rows == 0) return 0;
    const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const bool vec = width % 8 == 0 && width <= 512 * 8 * 4 && streams <= 4 && al(x) && al(x_new) && al(delta) &&
                     al(delta_bias) && al(gate) && al(gate_bias) && al(gain) && al(h) && al(shift) && al(shifted) && al(tail) &&
                     tail_stride % 4 == 0;
    int threads = vec ? 64 : (width >= 1024 ? 256 : 128);
    if (vec) while (threads < 512 && threads < width / 8) threads *= 2;
    // rows per block: one while the grid is short of the GPU, then runs, so that few rows are computed twice
    const int sms = sm_count_cached() > 0 ? sm_count_cached() : 148;
    const int resident = sms * (1024 / threads > 8 ? 8 : 1024 / threads);
    int run = 1;
    if (rows == nullptr && shift != nullptr) while (run < 8 && (long long)resident * run < n_rows) run *= 2;
    StreamArgs a{x, x_new, delta, delta_bias, gate, gate_bias, mix, out, in, gain, eps, h, shift, shifted, tail,
                 tail_stride, save_tails, token_slot, rows, n_rows, width, streams, run};
    const dim3 grid((n_rows + run - 1) / run), block(threads);
    if (vec) {
        const int per_thread = (width / 8 + threads - 1) / threads;
#define READ_SC(T, S, C) launch_pdl(kPdlNorm, stream_read_vec_kernel<T, S, C>, grid, block, 0, stream, a)
#define READ_S(T, S)                                    \
    do {                                                \
        if (per_thread <= 1) READ_SC(T, S, 1);          \
        else if (per_thread <= 2) READ_SC(T, S, 2);     \
        else READ_SC(T, S, 4);                          \
    } while (0)
#define READ(T)                                         \
    do {                                                \
        if (streams == 1) READ_S(T, 1);                 \
        else if (streams == 2) READ_S(T, 2);            \
        else if (streams == 3) READ_S(T, 3);            \
        else READ_S(T, 4);                              \
    } while (0)
        if (dtype == kBF16) READ(bf16);
        else READ(float);
#undef READ
#undef READ_S
#undef READ_SC
    } else {
        const size_t smem = (size_t)2 * width * sizeof(float);
        TLLM_REQUIRE(smem <= 200 * 1024, "stream_read: rows of %d elements are too wide", width);
        if (smem > 48 * 1024) {
            cudaError_t e = dtype == kBF16
                ? cudaFuncSetAttribute(stream_read_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
                : cudaFuncSetAttribute(stream_read_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) { set_error("stream_read: %s", cudaGetErrorString(e)); return (int)e; }
        }
        if (dtype == kBF16) launch_pdl(kPdlNorm, stream_read_kernel<bf16>, grid, block, smem, stream, a);
        else launch_pdl(kPdlNorm, stream_read_kernel<float>, grid, block, smem, stream, a);
    }
    return finish_launch("stream_read");
}

// seg_info: int[segments][4] = slot, first row, length, first position.
int tllm_stream_tails(const int* seg_info, int segments, const void* h, int dtype, float* tail, long long tail_stride,
                      int width, cudaStream_t stream) {
    TLLM_REQUIRE(segments >= 0 && width > 0 && seg_info && h && tail, "stream_tails: missing operand");
    if (segments == 0) return 0;
    const int threads = width >= 1024 ? 512 : 128;
    if (dtype == kBF16)
        launch_pdl(kPdlOther, stream_tails_kernel<bf16>, dim3(segments), dim3(threads), 0, stream, seg_info, (const bf16*)h, tail, tail_stride, width);
    else if (dtype == kF32)
        launch_pdl(kPdlOther, stream_tails_kernel<float>, dim3(segments), dim3(threads), 0, stream, seg_info, (const float*)h, tail, tail_stride, width);
    else TLLM_REQUIRE(false, "stream_tails: unknown dtype %d", dtype);
    return finish_launch("stream_tails");
}

// freq: float[ceil(width / 2)][2], a frequency and the rest of its rounding; out [tokens][streams][width].
int tllm_embedding_sinusoid(const int* ids, const int* positions, const void* table, int table_dtype, const float* freq,
                            float scale, float* out, int tokens, int width, int vocab, int streams, cudaStream_t stream) {
    TLLM_REQUIRE(tokens >= 0 && width > 0 && vocab > 0 && streams > 0, "embedding_sinusoid: bad sizes");
    TLLM_REQUIRE(ids && positions && table && freq && out, "embedding_sinusoid: missing operand");
    if (tokens == 0) return 0;
    const int threads = width >= 1024 ? 256 : 128;
    if (table_dtype == kBF16)
        launch_pdl(kPdlOther, embedding_sinusoid_kernel<bf16>, dim3(tokens), dim3(threads), 0, stream, ids, positions,
                   (const bf16*)table, (const float2*)freq, scale, out, width, vocab, streams);
    else if (table_dtype == kF32)
        launch_pdl(kPdlOther, embedding_sinusoid_kernel<float>, dim3(tokens), dim3(threads), 0, stream, ids, positions,
                   (const float*)table, (const float2*)freq, scale, out, width, vocab, streams);
    else TLLM_REQUIRE(false, "embedding_sinusoid: unknown dtype %d", table_dtype);
    return finish_launch("embedding_sinusoid");
}

}  // extern "C"
