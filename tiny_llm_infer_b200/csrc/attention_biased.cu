// Attention over the paged cache with a modified score: keys and values in planes of their own
// (their widths may differ), and between the dot product and the softmax any of
//   a cap          s <- cap * tanh(s / cap),
//   a distance bias s <- s - slope[head] * (pos_query - pos_key),
//   a chunk mask   keys only from the query's own chunk of `chunk` positions (counted from 0),
//   a window       keys pos - window + 1 .. pos,
//   a sink         one more term in the softmax's denominator that carries no value: exp(0), or exp(z_h) with a
//                  learned number z_h per query head (`sink_logit`; it is not scaled, capped or biased),
// and, instead of one attention map per head, the difference of two (`MAPS` = 2): a query head and a key head hold two
// vectors of width dk each, every map is a softmax of its own over the same values, and the head's result is
// a1 - lambda a2, divided by its root mean square over dv and times a constant (DiffMod);
// and after that an output gate: out *= sigmoid(gate).  Values may also be the first dv elements of
// wider rows (`v_row` elements from one value to the next; the attention over compressed vectors that serve
// as keys and, in part, as values passes the key plane twice).  Every constant is an argument; a
// zero (or a null pointer) switches its step off, and with all of them off this is plain causal
// attention.
//
// Four kernels.  `qkv_unit_store`: per-head RMS norm of queries and keys (with or without gains)
// and the write of keys and values into their pages.  `attention_biased_general`: one block per
// (token, query head), any widths up to 512, float32 or bfloat16; the float32 path and the fallback.
// `attention_biased_prefill`: bfloat16 prompt portions on mma.sync tiles, 64 query rows of one head
// per block, widths up to 128 (padded with zeros to 64 or 128 in shared memory).
// `attention_biased_decode`: one-token rows on the same tiles, one block per (row, key/value head, run of
// keys): the query heads of the group are the rows of the tile, so keys and values are read once for all.
//
// Scores, the cap, the bias, the softmax and the gate are float32 in both storage types.  The order of
// the additions for a (request, position, head) depends on the position and the constants only.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace tllm {

struct ScoreMod {
    float scale, softcap;
    int chunk, window, sink;
    const float* dist_bias;      // [query heads][dist_len] float32 added to the score by distance, or null
    int dist_len;                // distances from dist_len - 1 on share the last entry
    int gate_per_head;           // the output gate holds one number per query head instead of one per element
};

// Place of the gate of element e of a head within the token's gate row.
__device__ __forceinline__ size_t gate_at(int per_head, int head, int dv, int e) {
    return per_head ? (size_t)head : (size_t)head * dv + e;
}

// The learned bias of a head for a key `dist` tokens back (0 without a table).
__device__ __forceinline__ float dist_bias_of(const ScoreMod& m, int head, int dist) {
    if (m.dist_bias == nullptr) return 0.0f;
    return m.dist_bias[(size_t)head * m.dist_len + min(max(dist, 0), m.dist_len - 1)];
}

// The difference of two maps: o = a1 - lambda * a2, then o / sqrt(mean(o^2) + eps) * out_scale.
struct DiffMod {
    float lambda, eps, out_scale;
};

static inline int page_shift_of(int page_size) {
    int shift = 0;
    while ((1 << shift) < page_size) ++shift;
    return (1 << shift) == page_size ? shift : -1;
}

__device__ __forceinline__ int first_key(int pos, const ScoreMod& m) {
    int lo = 0;
    if (m.chunk > 0) lo = (pos / m.chunk) * m.chunk;
    if (m.window > 0 && pos - m.window + 1 > lo) lo = pos - m.window + 1;
    return lo;
}

__device__ __forceinline__ float mod_score(float dot, float slope, int dist, const ScoreMod& m) {
    float s = dot * m.scale;
    if (m.softcap > 0.0f) s = m.softcap * tanhf(s / m.softcap);
    return s - slope * (float)dist;
}

// ---------------------------------------------------------------- norm of q and k, write of k and v
// How queries and keys are normed: not at all, every head by itself (gains of dk numbers, shared by the heads), or
// all heads of a token together, the queries as one vector and the keys as another (gains of q_heads * dk and
// kv_heads * dk numbers).
enum QkNorm : int { kQkNone = 0, kQkPerHead = 1, kQkWhole = 2 };

// Values mixed with another layer's values of the same token, v <- keep v + share (first + first_bias), before they
// are written: `first` points at the token-0 row of those values as they were projected (heads side by side), `stride`
// elements from one token to the next.  Null: the values as they are.
template <typename T>
struct ValueMix {
    const T* first;
    int stride;
    const float* bias;
    float keep, share;
};

// Sums of squares of a token's queries and of its keys, each over all heads (every thread gets both).
template <typename F>
__device__ __forceinline__ void whole_sums(F square_sum, int q_len, int k_len, float* scratch, float& q_sum, float& k_sum) {
    q_sum = block_sum(square_sum(0, q_len), scratch);
    k_sum = block_sum(square_sum(q_len, q_len + k_len), scratch);
}

// proj[t] = q heads | k heads | v heads | (anything else).  One warp per head of a token.
template <typename T>
__global__ void qkv_unit_store_kernel(const T* proj, int row_stride, const T* __restrict__ q_gain,
                                      const T* __restrict__ k_gain, float eps, int do_norm,
                                      const int* __restrict__ positions, const int* __restrict__ token_slot,
                                      const int* __restrict__ block_table, int max_pages, int page_size,
                                      T* k_plane, T* v_plane, long long page_stride, T* q_out,
                                      int q_heads, int kv_heads, int dk, int dv, int store,
                                      const float* __restrict__ inv_freq, int rot_dims, int pairs, float temp_coef,
                                      int temp_every, int v_from_k, const float* __restrict__ bias, ValueMix<T> mix) {
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int pos = positions[t];
    const T* row = proj + (size_t)t * row_stride;
    // element c of the row as the kernel sees it: the projection plus its bias, if it has one, in float32
    auto at = [&](size_t c) -> float { return to_f32<T>(row[c]) + (bias != nullptr ? bias[c] : 0.0f); };
    long long page_base = -1;
    int in_page = 0;
    if (store) {
        const int page = block_table[(size_t)slot * max_pages + pos / page_size];
        page_base = (long long)page * page_stride;
        in_page = pos % page_size;
        if (page < 0) store = 0;          // no page held: nothing to write (the host reserves before a step)
    }
    const int total = q_heads + 2 * kv_heads;
    float q_whole = 1.0f, k_whole = 1.0f;
    if (do_norm == kQkWhole) {
        whole_sums([&](int from, int to) {
            float sum = 0.0f;
            for (int c = from + threadIdx.x; c < to; c += blockDim.x) { const float x = at(c); sum += x * x; }
            return sum;
        }, q_heads * dk, kv_heads * dk, scratch, q_whole, k_whole);
        q_whole = 1.0f / sqrtf(q_whole / (float)(q_heads * dk) + eps);
        k_whole = 1.0f / sqrtf(k_whole / (float)(kv_heads * dk) + eps);
    }
    for (int head = warp; head < total; head += warps) {
        if (head < q_heads + kv_heads) {
            const bool is_q = head < q_heads;
            const size_t src = (size_t)head * dk;
            const T* gain = is_q ? q_gain : k_gain;
            if (do_norm == kQkWhole && gain != nullptr) gain += (size_t)(is_q ? head : head - q_heads) * dk;
            float sc = is_q ? q_whole : k_whole;
            if (do_norm == kQkPerHead) {
                float sum = 0.0f;
                for (int e = lane; e < dk; e += 32) {
                    const float x = at(src + e);
                    sum += x * x;
                }
                sum = warp_sum(sum);
                sc = 1.0f / sqrtf(sum / (float)dk + eps);
            }
            T* dst;
            if (is_q) dst = q_out + ((size_t)t * q_heads + head) * dk;
            else if (store) dst = k_plane + page_base + ((size_t)(head - q_heads) * page_size + in_page) * dk;
            else continue;
            // a query's temperature grows with the logarithm of its position counted in runs of temp_every
            const float temp = (is_q && temp_every > 0) ? 1.0f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.0f) : 1.0f;
            const int half = rot_dims >> 1;
            for (int e = lane; e < dk; e += 32) {
                float x = at(src + e) * sc;
                if (gain != nullptr && do_norm) x *= to_f32<T>(gain[e]);
                if (e < rot_dims) {               // element e turns with its neighbour, or with its partner half a rotated width away
                    const bool low = pairs ? (e & 1) == 0 : e < half;
                    const int partner = pairs ? e ^ 1 : (low ? e + half : e - half);
                    float y = at(src + partner) * sc;
                    if (gain != nullptr && do_norm) y *= to_f32<T>(gain[partner]);
                    const float ang = (float)pos * inv_freq[pairs ? e >> 1 : (low ? e : e - half)];
                    const float c = cosf(ang), sn = sinf(ang);
                    x = low ? x * c - y * sn : x * c + y * sn;
                }
                dst[e] = from_f32<T>(x * temp);
            }
        } else if (store) {
            const int g = head - q_heads - kv_heads;
            // values of their own, or the keys as they were projected (before their norm)
            const size_t src = v_from_k ? (size_t)(q_heads + g) * dk
                                        : (size_t)(q_heads + kv_heads) * dk + (size_t)g * dv;
            T* dst = v_plane + page_base + ((size_t)g * page_size + in_page) * dv;
            if (mix.first != nullptr) {
                const T* other = mix.first + (size_t)t * mix.stride + (size_t)g * dv;
                for (int e = lane; e < dv; e += 32) {
                    const float f = to_f32<T>(other[e]) + (mix.bias != nullptr ? mix.bias[(size_t)g * dv + e] : 0.0f);
                    dst[e] = from_f32<T>(mix.keep * at(src + e) + mix.share * f);
                }
            } else if (bias != nullptr) for (int e = lane; e < dv; e += 32) dst[e] = from_f32<T>(at(src + e));
            else for (int e = lane; e < dv; e += 32) dst[e] = row[src + e];
        }
    }
}

// The same for bfloat16 rows whose widths are multiples of eight: a group of GS lanes (a power of two; dk / 8 of
// them at work) holds a head, eight elements to a lane, so a warp takes 32 / GS heads at once with 16-byte
// loads and stores.  The token's cosines and sines are made once, in shared memory, for all its heads; the
// partner of a rotated element sits half / 8 lanes away (half a multiple of eight) or, turning in neighbouring
// pairs, in the same lane.  The arithmetic per element is that of the kernel above.
__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}

template <int GS>
__global__ void __launch_bounds__(256)
qkv_unit_store_vec_kernel(const bf16* proj, int row_stride, const bf16* __restrict__ q_gain,
                          const bf16* __restrict__ k_gain, float eps, int do_norm,
                          const int* __restrict__ positions, const int* __restrict__ token_slot,
                          const int* __restrict__ block_table, int max_pages, int page_size, bf16* k_plane,
                          bf16* v_plane, long long page_stride, bf16* q_out, int q_heads, int kv_heads, int dk,
                          int dv, int store, const float* __restrict__ inv_freq, int rot_dims, int pairs, float temp_coef,
                          int temp_every, int v_from_k, const float* __restrict__ bias, ValueMix<bf16> mix) {
    extern __shared__ float cos_sin[];                      // cos of the token's `half` angles, then their sines
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;                                    // the whole block
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int pos = positions[t];
    const int half = rot_dims >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float ang = (float)pos * inv_freq[i];
        cos_sin[i] = cosf(ang);
        cos_sin[half + i] = sinf(ang);
    }
    if (half > 0) __syncthreads();
    const bf16* row = proj + (size_t)t * row_stride;
    long long page_base = -1;
    int in_page = 0;
    if (store) {
        const int page = block_table[(size_t)slot * max_pages + pos / page_size];
        page_base = (long long)page * page_stride;
        in_page = pos % page_size;
        if (page < 0) store = 0;
    }
    constexpr int kPerWarp = 32 / GS;
    const int grp = lane / GS, gl = lane % GS, e0 = gl * 8;
    const int normed = q_heads + kv_heads;
    const float q_temp = temp_every > 0 ? 1.0f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.0f) : 1.0f;
    // eight columns of the row as the kernel sees them: the projection plus its bias, if it has one, in float32
    auto at8 = [&](size_t c, float (&v)[8]) {
        load8(row + c, v);
        if (bias != nullptr) {
            const float4 b0 = *reinterpret_cast<const float4*>(bias + c);
            const float4 b1 = *reinterpret_cast<const float4*>(bias + c + 4);
            v[0] += b0.x; v[1] += b0.y; v[2] += b0.z; v[3] += b0.w;
            v[4] += b1.x; v[5] += b1.y; v[6] += b1.z; v[7] += b1.w;
        }
    };
    float q_whole = 1.0f, k_whole = 1.0f;
    if (do_norm == kQkWhole) {
        whole_sums([&](int from, int to) {
            float sum = 0.0f;
            for (int c = from + threadIdx.x * 8; c < to; c += blockDim.x * 8) {
                float v[8];
                at8(c, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) sum += v[e] * v[e];
            }
            return sum;
        }, q_heads * dk, kv_heads * dk, scratch, q_whole, k_whole);
        q_whole = 1.0f / sqrtf(q_whole / (float)(q_heads * dk) + eps);
        k_whole = 1.0f / sqrtf(k_whole / (float)(kv_heads * dk) + eps);
    }
    // with few rows a token's heads and values are dealt to gridDim.y blocks (which all make the sums over all heads)
    const int stride = gridDim.y * warps * kPerWarp;
    for (int base = (blockIdx.y * warps + warp) * kPerWarp; base < normed; base += stride) {
        const int head = base + grp;
        const bool is_q = head < q_heads;
        const bool active = head < normed && e0 < dk;
        float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
        if (active) at8((size_t)head * dk + e0, v);
        float sc = is_q ? q_whole : k_whole;
        if (do_norm == kQkPerHead) {
            float sum = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) sum += v[e] * v[e];
#pragma unroll
            for (int o = GS / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            sc = 1.0f / sqrtf(sum / (float)dk + eps);
        }
        const bf16* gain = is_q ? q_gain : k_gain;
        if (do_norm == kQkWhole && gain != nullptr) gain += (size_t)(is_q ? head : head - q_heads) * dk;
        if (active && gain != nullptr && do_norm) {
            float gn[8];
            load8(gain + e0, gn);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = v[e] * sc * gn[e];
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] *= sc;
        }
        if (pairs) {
#pragma unroll
            for (int e = 0; e < 8; e += 2) {
                if (e0 + e < rot_dims) {
                    const int i = (e0 + e) >> 1;
                    const float c = cos_sin[i], sn = cos_sin[half + i], x = v[e], y = v[e + 1];
                    v[e] = x * c - y * sn;
                    v[e + 1] = y * c + x * sn;
                }
            }
        } else if (half > 0) {                               // every lane takes part in the exchange
            const bool turns = e0 < rot_dims, low = e0 < half;
            const int from = turns ? (low ? lane + half / 8 : lane - half / 8) : lane;
            const int i0 = low ? e0 : e0 - half;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float y = __shfl_sync(0xffffffffu, v[e], from);
                if (turns) {
                    const float c = cos_sin[i0 + e], sn = cos_sin[half + i0 + e];
                    v[e] = low ? v[e] * c - y * sn : v[e] * c + y * sn;
                }
            }
        }
        if (!active) continue;
        bf16* dst;
        if (is_q) dst = q_out + ((size_t)t * q_heads + head) * dk;
        else if (store) dst = k_plane + page_base + ((size_t)(head - q_heads) * page_size + in_page) * dk;
        else continue;
        const float temp = is_q ? q_temp : 1.0f;
        uint4 raw;
        __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(v[2 * e] * temp, v[2 * e + 1] * temp);
        *reinterpret_cast<uint4*>(dst + e0) = raw;
    }
    if (store) {
        // values of their own, or the keys as they were projected (before their norm): 16 bytes a thread
        const int per_head = dv / 8;
        const bf16* src0 = v_from_k ? row + (size_t)q_heads * dk : row + (size_t)normed * dk;
        for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < kv_heads * per_head; c += gridDim.y * blockDim.x) {
            const int g = c / per_head, j = c - g * per_head;
            bf16* dst = v_plane + page_base + ((size_t)g * page_size + in_page) * dv + j * 8;
            if (bias == nullptr && mix.first == nullptr) {
                *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src0 + (size_t)g * dv + j * 8);
                continue;
            }
            float v[8];
            at8((src0 - row) + (size_t)g * dv + j * 8, v);
            if (mix.first != nullptr) {
                float f[8];
                load8(mix.first + (size_t)t * mix.stride + (size_t)g * dv + j * 8, f);
                const float* b = mix.bias != nullptr ? mix.bias + (size_t)g * dv + j * 8 : nullptr;
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = mix.keep * v[e] + mix.share * (f[e] + (b != nullptr ? b[e] : 0.0f));
            }
            uint4 raw;
            __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
            *reinterpret_cast<uint4*>(dst) = raw;
        }
    }
}

// ---------------------------------------------------------------- general kernel
constexpr int kGenWarps = 4;

template <typename T, int CK, int CV, int MAPS>
__global__ void attention_biased_general_kernel(
    const T* q, const T* k_plane, const T* v_plane, long long page_stride,
    const int* __restrict__ positions, const int* __restrict__ token_slot,
    const int* __restrict__ block_table, int max_pages, int page_size, int q_heads, int kv_heads,
    int dk, int dv, ScoreMod mod, DiffMod diff, const float* __restrict__ slopes, const float* __restrict__ sink_logit, int v_row,
    const T* gate, int gate_stride, T* __restrict__ out) {
    extern __shared__ float smem[];
    __shared__ float scratch[32];
    TLLM_PDL_ENTER();
    const int kd = MAPS * dk;                     // elements of a query head and of a cached key
    float* qs = smem;                             // [MAPS][dk]
    float* acc_s = smem + kd;                     // [MAPS][warps][dv]
    float* m_s = acc_s + MAPS * kGenWarps * dv;   // [MAPS][warps]
    float* l_s = m_s + MAPS * kGenWarps;          // [MAPS][warps]

    const int head = blockIdx.x, t = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    T* dst = out + ((size_t)t * q_heads + head) * dv;
    const int slot = token_slot[t];
    if (slot < 0) {
        for (int e = threadIdx.x; e < dv; e += blockDim.x) dst[e] = from_f32<T>(0.0f);
        return;
    }
    const int pos = positions[t];
    const int lo = first_key(pos, mod);
    const int g = head / (q_heads / kv_heads);
    const float slope = slopes != nullptr ? slopes[head] : 0.0f;
    const T* qsrc = q + ((size_t)t * q_heads + head) * kd;
    for (int e = threadIdx.x; e < kd; e += blockDim.x) qs[e] = to_f32<T>(qsrc[e]);
    __syncthreads();

    const int* table = block_table + (size_t)slot * max_pages;
    // the sink is a key of score 0 (or of the head's learned score) without a value; warp 0 starts from it
    float m[MAPS], l[MAPS], acc[MAPS][CV];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        m[mp] = (mod.sink && warp == 0) ? (sink_logit != nullptr ? sink_logit[head] : 0.0f) : -INFINITY;
        l[mp] = (mod.sink && warp == 0) ? 1.0f : 0.0f;
#pragma unroll
        for (int c = 0; c < CV; ++c) acc[mp][c] = 0.0f;
    }

    for (int j = lo + warp; j <= pos; j += kGenWarps) {
        const int page = table[j / page_size];
        if (page < 0) continue;
        const size_t in_page = (size_t)g * page_size + (j % page_size);
        const T* kp = k_plane + (long long)page * page_stride + in_page * kd;
        const T* vp = v_plane + (long long)page * page_stride + in_page * v_row;
#pragma unroll
        for (int mp = 0; mp < MAPS; ++mp) {
            float dot = 0.0f;
#pragma unroll
            for (int c = 0; c < CK; ++c) {
                const int e = lane + 32 * c;
                if (e < dk) dot += qs[mp * dk + e] * to_f32<T>(kp[mp * dk + e]);
            }
            dot = warp_sum(dot);
            const float s = mod_score(dot, slope, pos - j, mod) + dist_bias_of(mod, head, pos - j);
            const float m_new = fmaxf(m[mp], s);
            const float corr = expf(m[mp] - m_new);
            const float p = expf(s - m_new);
            l[mp] = l[mp] * corr + p;
#pragma unroll
            for (int c = 0; c < CV; ++c) {
                const int e = lane + 32 * c;
                if (e < dv) acc[mp][c] = acc[mp][c] * corr + p * to_f32<T>(vp[e]);
            }
            m[mp] = m_new;
        }
    }
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        if (lane == 0) { m_s[mp * kGenWarps + warp] = m[mp]; l_s[mp * kGenWarps + warp] = l[mp]; }
#pragma unroll
        for (int c = 0; c < CV; ++c) {
            const int e = lane + 32 * c;
            if (e < dv) acc_s[(mp * kGenWarps + warp) * dv + e] = acc[mp][c];
        }
    }
    __syncthreads();
    float w_scale[MAPS][kGenWarps];               // a warp's share of a map's result, its sum divided out
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        float mm = m_s[mp * kGenWarps], total = 0.0f;
#pragma unroll
        for (int w = 1; w < kGenWarps; ++w) mm = fmaxf(mm, m_s[mp * kGenWarps + w]);
#pragma unroll
        for (int w = 0; w < kGenWarps; ++w) {
            w_scale[mp][w] = (m_s[mp * kGenWarps + w] == -INFINITY) ? 0.0f : expf(m_s[mp * kGenWarps + w] - mm);
            total += l_s[mp * kGenWarps + w] * w_scale[mp][w];
        }
        const float inv = total > 0.0f ? 1.0f / total : 0.0f;
        if (MAPS > 1) {
#pragma unroll
            for (int w = 0; w < kGenWarps; ++w) w_scale[mp][w] *= mp == 0 ? inv : -diff.lambda * inv;
        } else {
            m[0] = inv;                           // one map: the sum over the warps is taken first
        }
    }
    float norm = 1.0f;
    if (MAPS > 1) {
        float sum = 0.0f;
        for (int e = threadIdx.x; e < dv; e += blockDim.x) {
            float v = 0.0f;
#pragma unroll
            for (int mp = 0; mp < MAPS; ++mp)
#pragma unroll
                for (int w = 0; w < kGenWarps; ++w) v += acc_s[(mp * kGenWarps + w) * dv + e] * w_scale[mp][w];
            acc_s[e] = v;                         // only this thread looks at column e
            sum += v * v;
        }
        norm = diff.out_scale / sqrtf(block_sum(sum, scratch) / (float)dv + diff.eps);
    }
    const T* grow = gate != nullptr ? gate + (size_t)t * gate_stride + gate_at(mod.gate_per_head, head, dv, 0) : nullptr;
    for (int e = threadIdx.x; e < dv; e += blockDim.x) {
        float v = 0.0f;
        if (MAPS > 1) {
            v = acc_s[e] * norm;
        } else {
#pragma unroll
            for (int w = 0; w < kGenWarps; ++w) v += acc_s[w * dv + e] * w_scale[0][w];
            v *= m[0];
        }
        if (grow != nullptr) v *= 1.0f / (1.0f + expf(-to_f32<T>(grow[mod.gate_per_head ? 0 : e])));
        dst[e] = from_f32<T>(v);
    }
}

template <typename T, int MAPS>
static int launch_general(const void* q, const void* kp, const void* vp, long long page_stride,
                          const int* positions, const int* token_slot, const int* block_table,
                          int max_pages, int page_size, int tokens, int q_heads, int kv_heads, int dk,
                          int dv, ScoreMod mod, DiffMod diff, const float* slopes, const float* sink_logit, int v_row,
                          const void* gate, int gate_stride, void* out, cudaStream_t stream) {
    const dim3 grid(q_heads, tokens), block(kGenWarps * 32);
    const size_t smem = (size_t)MAPS * ((size_t)dk + (size_t)kGenWarps * dv + 2 * kGenWarps) * sizeof(float);
    const int ck = (dk + 31) / 32, cv = (dv + 31) / 32;
    const int c = ck > cv ? ck : cv;
#define LAUNCH(C)                                                                                           \
    launch_pdl(kPdlAttention, attention_biased_general_kernel<T, C, C, MAPS>, grid, block, smem, stream,          \
               (const T*)q, (const T*)kp, (const T*)vp, page_stride, positions, token_slot, block_table,    \
               max_pages, page_size, q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row, (const T*)gate, gate_stride, (T*)out)
    if (c <= 1) LAUNCH(1);
    else if (c <= 2) LAUNCH(2);
    else if (c <= 4) LAUNCH(4);
    else if (c <= 8) LAUNCH(8);
    else LAUNCH(16);
#undef LAUNCH
    return finish_launch("attention_biased_general");
}

constexpr float kLog2e = 1.4426950408889634f;

// tanh(x) = 1 - 2 / (e^2x + 1): absolute error of a few 1e-7 with the fast exponential and division,
// which the cap multiplies; |x| is clamped where tanh is 1 to the last bit anyway.
__device__ __forceinline__ float fast_tanh(float x) {
    x = fminf(fmaxf(x, -15.0f), 15.0f);
    return 1.0f - __fdividef(2.0f, __expf(2.0f * x) + 1.0f);
}

// 2^x by the hardware approximation alone (exp2f adds a range reduction for denormal results; here a
// weight that small is zero anyway).  2^-inf = 0.
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Page and place in the page of a key: a shift and a mask where the page size is a power of two
// (`shift` >= 0), else a division.
__device__ __forceinline__ void page_of(int key, int page_size, int shift, int& page_index, int& in_page) {
    if (shift >= 0) { page_index = key >> shift; in_page = key & (page_size - 1); }
    else { page_index = key / page_size; in_page = key - page_index * page_size; }
}

// The modified score times log2(e), for exp2f.  `dist` comes as a float and 1 / cap as a factor: a
// conversion or a division per score would go through the same slow unit as the exponentials.  No
// branch: the capped and the plain score are both made and one is kept, so that the scores of a tile
// are independent chains the scheduler can interleave (with the mask as a condition around the
// arithmetic every score was a branch of its own, and the chains ran one after the other).
__device__ __forceinline__ float mod_score_fast(float dot, float slope_log2e, float dist, const ScoreMod& m, float inv_cap) {
    const float plain = dot * m.scale;
    const float capped = m.softcap * fast_tanh(plain * inv_cap);
    const float s = m.softcap > 0.0f ? capped : plain;
    return s * kLog2e - slope_log2e * dist;
}

// ---------------------------------------------------------------- prompt portions, bfloat16, mma.sync
// A block owns 64 consecutive query rows of one portion and one query head and walks the keys its rows
// can see in tiles of 64 (flash-attention style: S and the softmax in float32 registers, P V accumulated
// in float32).  Keys and values are staged by cp.async in two buffers; a row of a tile is padded by 16
// bytes so that ldmatrix meets no bank conflict, and widths below DKP / DVP are filled with zeros.
// With two maps a block owns 32 query rows: two of its warps hold them for the first map, two for the second, all
// share the tiles (a key row holds both maps' keys), and the maps meet in shared memory at the end.
constexpr int kPfWarps = 4, kPfM = 64, kPfN = 64, kPfPad = 8;

template <int DKP, int DVP, int MAPS>
__global__ void __launch_bounds__(kPfWarps * 32, 3)
attention_biased_prefill_kernel(const bf16* q, const bf16* k_plane, const bf16* v_plane, long long page_stride,
                                const int* __restrict__ seg_info, const int* __restrict__ tiles,
                                const int* __restrict__ block_table, int max_pages, int page_size,
                                int page_shift, int q_heads, int kv_heads, int dk, int dv, ScoreMod mod, DiffMod diff,
                                const float* __restrict__ slopes, const float* __restrict__ sink_logit, int v_row,
                                const bf16* gate, int gate_stride, bf16* __restrict__ out) {
    extern __shared__ __align__(128) unsigned char pf_smem[];
    TLLM_PDL_ENTER();
    constexpr int kKRow = MAPS * DKP + kPfPad, kVRow = DVP + kPfPad;    // elements per padded row
    constexpr int kKBytes = kPfN * kKRow * 2, kVBytes = kPfN * kVRow * 2;
    constexpr int kRows = kPfM / MAPS, kMapWarps = kPfWarps / MAPS;     // query rows of the block, warps per map
    const int kd = MAPS * dk;                                           // elements of a query head and of a cached key
    const int seg = tiles[2 * blockIdx.x], q_off = tiles[2 * blockIdx.x + 1] + (MAPS > 1 ? (int)blockIdx.z * kRows : 0);
    const int head = blockIdx.y;
    const int slot = seg_info[4 * seg], start = seg_info[4 * seg + 1];
    const int len = seg_info[4 * seg + 2], pos0 = seg_info[4 * seg + 3];
    if (MAPS > 1 && q_off >= len) return;                               // the second half of a block of 64 rows may be empty
    const int lane = threadIdx.x & 31, map = (threadIdx.x >> 5) / kMapWarps;
    const int warp = (threadIdx.x >> 5) % kMapWarps;                    // among the warps of the map
    const int g = head / (q_heads / kv_heads);
    const int* table = block_table + (size_t)slot * max_pages;
    const float slope2 = (slopes != nullptr ? slopes[head] : 0.0f) * kLog2e;
    const float inv_cap = mod.softcap > 0.0f ? 1.0f / mod.softcap : 0.0f;

    const int rows_here = min(kRows, len - q_off);
    const int first_pos = pos0 + q_off, last_pos = first_pos + rows_here - 1;
    const int lo_all = first_key(first_pos, mod);
    const int kt_first = lo_all / kPfN, kt_last = last_pos / kPfN;

    const int r_lo = warp * 16 + (lane >> 2), r_hi = r_lo + 8;
    const bool v_lo = r_lo < rows_here, v_hi = r_hi < rows_here;
    const int p_lo = first_pos + r_lo, p_hi = first_pos + r_hi;
    const int f_lo = first_key(p_lo, mod), f_hi = first_key(p_hi, mod);
    const bf16* q_lo = q + ((size_t)(start + q_off + r_lo) * q_heads + head) * kd + map * dk;
    const bf16* q_hi = q + ((size_t)(start + q_off + r_hi) * q_heads + head) * kd + map * dk;
    uint32_t qa[DKP / 16][4];
#pragma unroll
    for (int ks = 0; ks < DKP / 16; ++ks) {
        const int c0 = ks * 16 + (lane & 3) * 2;
        qa[ks][0] = (v_lo && c0 < dk) ? *reinterpret_cast<const uint32_t*>(q_lo + c0) : 0u;
        qa[ks][1] = (v_hi && c0 < dk) ? *reinterpret_cast<const uint32_t*>(q_hi + c0) : 0u;
        qa[ks][2] = (v_lo && c0 + 8 < dk) ? *reinterpret_cast<const uint32_t*>(q_lo + c0 + 8) : 0u;
        qa[ks][3] = (v_hi && c0 + 8 < dk) ? *reinterpret_cast<const uint32_t*>(q_hi + c0 + 8) : 0u;
    }
    const int w_first = first_pos + warp * 16;
    const int w_last = min(w_first + 15, last_pos);
    const int w_lo = first_key(w_first, mod);
    const int w_hi_lo = first_key(w_first + 15, mod);                  // the latest first key among the warp's rows

    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    // the sink: a key of score 0 (or the head's learned score) without a value, counted once per row (by the
    // first lane of its four)
    float m_lo = mod.sink ? (sink_logit != nullptr ? sink_logit[head] * kLog2e : 0.0f) : -INFINITY, m_hi = m_lo;
    float l_lo = (mod.sink && (lane & 3) == 0) ? 1.0f : 0.0f, l_hi = l_lo;

    auto issue = [&](int kt, int stage) {
        const uint32_t ks = smem_u32(pf_smem + (size_t)stage * (kKBytes + kVBytes));
        const uint32_t vs = ks + kKBytes;
        constexpr int kMC = DKP / 8, kKC = MAPS * kMC, kVC = DVP / 8;       // 16-byte pieces of a map's key, a row of keys, a value
        // a thread keeps its 16-byte column and walks the rows: one look-up of the page per row
        for (int row = threadIdx.x / kKC, chunk = threadIdx.x % kKC; row < kPfN; row += kPfWarps * 32 / kKC) {
            const int key = kt * kPfN + row;
            int page_index, place;
            page_of(key, page_size, page_shift, page_index, place);
            const int page = (key <= last_pos && key >= lo_all) ? table[page_index] : -1;
            const bool ok = page >= 0;
            const long long page_at = ok ? (long long)page * page_stride : 0;
            const long long in_page = (long long)g * page_size + place;
            const int in_key = (chunk % kMC) * 8;                       // within its map's key
            const bool k_ok = ok && in_key < dk;
            cp_async_16(ks + (row * kKRow + chunk * 8) * 2, k_plane + (k_ok ? page_at + in_page * kd + (chunk / kMC) * dk + in_key : 0), k_ok);
            if (kKC == kVC) {
                const bool v_ok = ok && chunk * 8 < dv;
                cp_async_16(vs + (row * kVRow + chunk * 8) * 2, v_plane + (v_ok ? page_at + in_page * v_row + chunk * 8 : 0), v_ok);
            }
        }
        if (kKC != kVC) {
            for (int row = threadIdx.x / kVC, chunk = threadIdx.x % kVC; row < kPfN; row += kPfWarps * 32 / kVC) {
                const int key = kt * kPfN + row;
                int page_index, place;
                page_of(key, page_size, page_shift, page_index, place);
                const int page = (key <= last_pos && key >= lo_all) ? table[page_index] : -1;
                const bool v_ok = page >= 0 && chunk * 8 < dv;
                cp_async_16(vs + (row * kVRow + chunk * 8) * 2, v_plane + (v_ok ? (long long)page * page_stride + ((long long)g * page_size + place) * v_row + chunk * 8 : 0), v_ok);
            }
        }
        cp_async_commit();
    };

    issue(kt_first, 0);
    for (int kt = kt_first; kt <= kt_last; ++kt) {
        const int stage = (kt - kt_first) & 1;
        if (kt + 1 <= kt_last) {
            issue(kt + 1, stage ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int key0 = kt * kPfN;
        const bool active = warp * 16 < rows_here && key0 <= w_last && key0 + kPfN - 1 >= w_lo;
        if (active) {
            const uint32_t ks_base = smem_u32(pf_smem + (size_t)stage * (kKBytes + kVBytes));
            const uint32_t vs_base = ks_base + kKBytes;
            const int mid = lane >> 3, mrow = lane & 7;
            float s[kPfN / 8][4];
#pragma unroll
            for (int i = 0; i < kPfN / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
            for (int ks = 0; ks < DKP / 16; ++ks) {               // columns past dk are zeros on both sides
#pragma unroll
                for (int nt2 = 0; nt2 < kPfN / 16; ++nt2) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, ks_base + ((nt2 * 16 + (mid >> 1) * 8 + mrow) * kKRow + map * DKP + ks * 16 + (mid & 1) * 8) * 2);
                    const uint32_t b0[2] = {kb[0], kb[1]}, b1[2] = {kb[2], kb[3]};
                    mma_bf16_16816(s[2 * nt2], qa[ks], b0);
                    mma_bf16_16816(s[2 * nt2 + 1], qa[ks], b1);
                }
            }
            const int key_base = key0 + (lane & 3) * 2;
            const float d_lo = (float)(p_lo - key_base), d_hi = (float)(p_hi - key_base);
            // a tile that every row of the warp sees whole needs no masks (most tiles of a long prompt)
            const bool inner = key0 + kPfN - 1 <= w_first && key0 >= w_hi_lo;
            float tmax_lo = -INFINITY, tmax_hi = -INFINITY;
#pragma unroll
            for (int nt = 0; nt < kPfN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float back = (float)(nt * 8 + e);          // a constant once the loops are unrolled
                    s[nt][e] = mod_score_fast(s[nt][e], slope2, d_lo - back, mod, inv_cap);
                    s[nt][2 + e] = mod_score_fast(s[nt][2 + e], slope2, d_hi - back, mod, inv_cap);
                }
            if (mod.dist_bias != nullptr) {
                // a tile that lies beyond the table for every row of the warp gets the table's last entry;
                // only the few tiles near the diagonal look distances up one by one
                const float* tb = mod.dist_bias + (size_t)head * mod.dist_len;
                const int lastd = mod.dist_len - 1;
                if (first_pos + warp * 16 - (key0 + kPfN - 1) >= lastd) {
                    const float far = tb[lastd] * kLog2e;
#pragma unroll
                    for (int nt = 0; nt < kPfN / 8; ++nt) { s[nt][0] += far; s[nt][1] += far; s[nt][2] += far; s[nt][3] += far; }
                } else {
                    const int n_lo = p_lo - key_base, n_hi = p_hi - key_base;
#pragma unroll
                    for (int nt = 0; nt < kPfN / 8; ++nt)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            s[nt][e] += tb[min(max(n_lo - (nt * 8 + e), 0), lastd)] * kLog2e;
                            s[nt][2 + e] += tb[min(max(n_hi - (nt * 8 + e), 0), lastd)] * kLog2e;
                        }
                }
            }
            if (!inner) {
#pragma unroll
                for (int nt = 0; nt < kPfN / 8; ++nt)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int j = key_base + nt * 8 + e;
                        s[nt][e] = (j <= p_lo && j >= f_lo) ? s[nt][e] : -INFINITY;
                        s[nt][2 + e] = (j <= p_hi && j >= f_hi) ? s[nt][2 + e] : -INFINITY;
                    }
            }
#pragma unroll
            for (int nt = 0; nt < kPfN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    tmax_lo = fmaxf(tmax_lo, s[nt][e]);
                    tmax_hi = fmaxf(tmax_hi, s[nt][2 + e]);
                }
            tmax_lo = fmaxf(tmax_lo, __shfl_xor_sync(0xffffffffu, tmax_lo, 1));
            tmax_lo = fmaxf(tmax_lo, __shfl_xor_sync(0xffffffffu, tmax_lo, 2));
            tmax_hi = fmaxf(tmax_hi, __shfl_xor_sync(0xffffffffu, tmax_hi, 1));
            tmax_hi = fmaxf(tmax_hi, __shfl_xor_sync(0xffffffffu, tmax_hi, 2));
            const float mn_lo = fmaxf(m_lo, tmax_lo), mn_hi = fmaxf(m_hi, tmax_hi);
            const float ms_lo = mn_lo == -INFINITY ? 0.0f : mn_lo, ms_hi = mn_hi == -INFINITY ? 0.0f : mn_hi;
            const float c_lo = fast_exp2(m_lo - ms_lo), c_hi = fast_exp2(m_hi - ms_hi);
            m_lo = mn_lo;
            m_hi = mn_hi;
            float sum_lo = 0.0f, sum_hi = 0.0f;
#pragma unroll
            for (int nt = 0; nt < kPfN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    s[nt][e] = fast_exp2(s[nt][e] - ms_lo);
                    s[nt][2 + e] = fast_exp2(s[nt][2 + e] - ms_hi);
                    sum_lo += s[nt][e];
                    sum_hi += s[nt][2 + e];
                }
            l_lo = l_lo * c_lo + sum_lo;
            l_hi = l_hi * c_hi + sum_hi;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) {
                o[i][0] *= c_lo; o[i][1] *= c_lo; o[i][2] *= c_hi; o[i][3] *= c_hi;
            }
#pragma unroll
            for (int kk = 0; kk < kPfN / 16; ++kk) {
                const uint32_t pa[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                        pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]),
                                        pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                for (int c = 0; c < DVP / 8; c += 2) {             // value columns past dv are zeros
                    uint32_t vb[4];
                    ldmatrix_x4_trans(vb, vs_base + ((kk * 16 + (mid & 1) * 8 + mrow) * kVRow + (c + (mid >> 1)) * 8) * 2);
                    const uint32_t b0[2] = {vb[0], vb[1]}, b1[2] = {vb[2], vb[3]};
                    mma_bf16_16816(o[c], pa, b0);
                    mma_bf16_16816(o[c + 1], pa, b1);
                }
            }
        }
        __syncthreads();
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    float inv_lo = l_lo > 0.0f ? 1.0f / l_lo : 0.0f, inv_hi = l_hi > 0.0f ? 1.0f / l_hi : 0.0f;
    const size_t row_lo = start + q_off + r_lo, row_hi = start + q_off + r_hi;
    if (MAPS > 1) {
        // the second map's rows, times lambda, in shared memory (over the tiles, which every warp is done with); the
        // first map's warps take them off their own, and a row's four lanes add up its squares
        float* meet = reinterpret_cast<float*>(pf_smem);                 // [kRows][DVP + 2]
        constexpr int kMeet = DVP + 2;
        if (map == 1) {
            const float a_lo = inv_lo * diff.lambda, a_hi = inv_hi * diff.lambda;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) {
                const int col = i * 8 + (lane & 3) * 2;
                *reinterpret_cast<float2*>(meet + r_lo * kMeet + col) = make_float2(o[i][0] * a_lo, o[i][1] * a_lo);
                *reinterpret_cast<float2*>(meet + r_hi * kMeet + col) = make_float2(o[i][2] * a_hi, o[i][3] * a_hi);
            }
        }
        __syncthreads();
        if (map == 1) return;
        float sq_lo = 0.0f, sq_hi = 0.0f;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) {                              // columns past dv are zeros in both maps
            const int col = i * 8 + (lane & 3) * 2;
            const float2 b_lo = *reinterpret_cast<const float2*>(meet + r_lo * kMeet + col);
            const float2 b_hi = *reinterpret_cast<const float2*>(meet + r_hi * kMeet + col);
            o[i][0] = o[i][0] * inv_lo - b_lo.x; o[i][1] = o[i][1] * inv_lo - b_lo.y;
            o[i][2] = o[i][2] * inv_hi - b_hi.x; o[i][3] = o[i][3] * inv_hi - b_hi.y;
            sq_lo += o[i][0] * o[i][0] + o[i][1] * o[i][1];
            sq_hi += o[i][2] * o[i][2] + o[i][3] * o[i][3];
        }
        sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 1);
        sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 2);
        sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 1);
        sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 2);
        inv_lo = diff.out_scale / sqrtf(sq_lo / (float)dv + diff.eps);
        inv_hi = diff.out_scale / sqrtf(sq_hi / (float)dv + diff.eps);
    }
    bf16* o_lo = out + (row_lo * q_heads + head) * dv;
    bf16* o_hi = out + (row_hi * q_heads + head) * dv;
    const bf16* g_lo = gate != nullptr ? gate + row_lo * gate_stride + gate_at(mod.gate_per_head, head, dv, 0) : nullptr;
    const bf16* g_hi = gate != nullptr ? gate + row_hi * gate_stride + gate_at(mod.gate_per_head, head, dv, 0) : nullptr;
    const int g_step = mod.gate_per_head ? 0 : 1;
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) {
        const int col = i * 8 + (lane & 3) * 2;
        if (col >= dv) continue;
        if (v_lo) {
            float a = o[i][0] * inv_lo, b = o[i][1] * inv_lo;
            if (g_lo != nullptr) {
                a *= 1.0f / (1.0f + expf(-__bfloat162float(g_lo[col * g_step])));
                b *= 1.0f / (1.0f + expf(-__bfloat162float(g_lo[(col + 1) * g_step])));
            }
            *reinterpret_cast<uint32_t*>(o_lo + col) = pack_bf16(a, b);
        }
        if (v_hi) {
            float a = o[i][2] * inv_hi, b = o[i][3] * inv_hi;
            if (g_hi != nullptr) {
                a *= 1.0f / (1.0f + expf(-__bfloat162float(g_hi[col * g_step])));
                b *= 1.0f / (1.0f + expf(-__bfloat162float(g_hi[(col + 1) * g_step])));
            }
            *reinterpret_cast<uint32_t*>(o_hi + col) = pack_bf16(a, b);
        }
    }
}

template <int DKP, int DVP, int MAPS>
static int launch_biased_prefill(const void* q, const void* kp, const void* vp, long long page_stride,
                                 const int* seg_info, const int* tiles, int n_tiles, const int* block_table,
                                 int max_pages, int page_size, int q_heads, int kv_heads, int dk, int dv,
                                 ScoreMod mod, DiffMod diff, const float* slopes, const float* sink_logit, int v_row, const void* gate,
                                 int gate_stride, void* out, cudaStream_t stream) {
    const size_t smem = (size_t)2 * kPfN * ((MAPS * DKP + kPfPad) + (DVP + kPfPad)) * 2;
    static OncePerDevice configured;
    if (configured.first()) {
        cudaError_t e = cudaFuncSetAttribute(attention_biased_prefill_kernel<DKP, DVP, MAPS>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { set_error("attention_biased_prefill: %s", cudaGetErrorString(e)); return (int)e; }
        configured.done();
    }
    launch_pdl(kPdlAttention, attention_biased_prefill_kernel<DKP, DVP, MAPS>, dim3(n_tiles, q_heads, MAPS), dim3(kPfWarps * 32),
               smem, stream, (const bf16*)q, (const bf16*)kp, (const bf16*)vp, page_stride, seg_info, tiles,
               block_table, max_pages, page_size, page_shift_of(page_size), q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row,
               (const bf16*)gate, gate_stride, (bf16*)out);
    return finish_launch("attention_biased_prefill");
}

// ---------------------------------------------------------------- one-token rows, bfloat16, mma.sync
// One block per (row, key/value head, run of keys) (per sixteen query heads of it, if it serves more).  The query heads of the group are the 16 rows of the
// tensor-core tile (the first `group` of them real), so keys and values are read once for all of them.
// The block stages tiles of 64 keys like the prompt kernel; each of its four warps takes 16 keys of a
// tile and keeps its own running maximum, sum and value sums (base 2), which meet in shared memory in
// the order of the warps.  With one run per row the block writes the result; with more (a grid that
// would not fill the GPU, long reaches) it leaves unnormalised sums, maximum and weight per run, and a
// second kernel adds the runs in their order.  The sink belongs to the first warp of the first run.
// With two maps a tile's rows are the group's heads for the first map, then the same heads for the second; a row's
// query is its map's half of a vector as wide as a row of keys (both maps' keys side by side), the other half zeros,
// so that one product serves both maps and keys and values are still read once.
template <int DKP, int DVP, int MAPS>
__global__ void __launch_bounds__(kPfWarps * 32, 2)
attention_biased_decode_kernel(const bf16* q, const bf16* k_plane, const bf16* v_plane, long long page_stride,
                               const int* __restrict__ positions, const int* __restrict__ token_slot,
                               const int* __restrict__ rows, const int* __restrict__ block_table, int max_pages,
                               int page_size, int page_shift, int q_heads, int kv_heads, int dk, int dv, ScoreMod mod,
                               DiffMod diff, const float* __restrict__ slopes, const float* __restrict__ sink_logit, int v_row,
                               const bf16* gate, int gate_stride, int splits, int sub_groups, float* part,
                               bf16* __restrict__ out) {
    extern __shared__ __align__(128) unsigned char pf_smem[];
    TLLM_PDL_ENTER();
    constexpr int kKRow = MAPS * DKP + kPfPad, kVRow = DVP + kPfPad;
    const int kd = MAPS * dk;                                           // elements of a query head and of a cached key
    constexpr int kKBytes = kPfN * kKRow * 2, kVBytes = kPfN * kVRow * 2;
    const int t = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
    // a key/value head's query heads fill the tile's 16 rows; more of them (multi-query attention over many
    // heads) are dealt to `sub_groups` blocks that read the same keys
    const int g = blockIdx.y / sub_groups, split = blockIdx.z;
    const int group = q_heads / kv_heads / sub_groups;
    const int head0 = g * (q_heads / kv_heads) + (blockIdx.y % sub_groups) * group;
    const int slot = token_slot[t];
    const int rec = dv + 2;
    if (slot < 0) {
        if (splits == 1)
            for (int i = threadIdx.x; i < group * dv; i += blockDim.x)
                out[((size_t)t * q_heads + head0) * dv + i] = __float2bfloat16_rn(0.0f);
        return;                       // the combining kernel writes the zeros of a row without a request
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = positions[t];
    const int lo = first_key(pos, mod);
    const int* table = block_table + (size_t)slot * max_pages;
    int kt_first = lo / kPfN, kt_last = pos / kPfN;
    if (splits > 1) {
        const int per = (kt_last - kt_first + splits) / splits;
        kt_first += split * per;
        kt_last = min(kt_last, kt_first + per - 1);
    }

    const int r_lo = lane >> 2, r_hi = r_lo + 8;                       // rows of the tile: heads of the group (per map)
    const int used = MAPS * group;
    const bool v_lo = r_lo < used, v_hi = r_hi < used;
    const int map_lo = MAPS > 1 && r_lo >= group ? 1 : 0, map_hi = MAPS > 1 && r_hi >= group ? 1 : 0;
    const int h_lo = r_lo - map_lo * group, h_hi = r_hi - map_hi * group;          // heads of the group that the rows are
    const float slope_lo = (slopes != nullptr && v_lo) ? slopes[head0 + h_lo] * kLog2e : 0.0f;
    const float slope_hi = (slopes != nullptr && v_hi) ? slopes[head0 + h_hi] * kLog2e : 0.0f;
    const float inv_cap = mod.softcap > 0.0f ? 1.0f / mod.softcap : 0.0f;
    const bf16* q_lo = q + ((size_t)t * q_heads + head0 + h_lo) * kd + map_lo * dk;
    const bf16* q_hi = q + ((size_t)t * q_heads + head0 + h_hi) * kd + map_hi * dk;
    uint32_t qa[MAPS * DKP / 16][4];
#pragma unroll
    for (int ks = 0; ks < MAPS * DKP / 16; ++ks) {
        const int mk = ks / (DKP / 16);                                 // the map whose keys these columns are
        const int c0 = (ks - mk * (DKP / 16)) * 16 + (lane & 3) * 2;
        const bool w_lo = v_lo && map_lo == mk, w_hi = v_hi && map_hi == mk;
        qa[ks][0] = (w_lo && c0 < dk) ? *reinterpret_cast<const uint32_t*>(q_lo + c0) : 0u;
        qa[ks][1] = (w_hi && c0 < dk) ? *reinterpret_cast<const uint32_t*>(q_hi + c0) : 0u;
        qa[ks][2] = (w_lo && c0 + 8 < dk) ? *reinterpret_cast<const uint32_t*>(q_lo + c0 + 8) : 0u;
        qa[ks][3] = (w_hi && c0 + 8 < dk) ? *reinterpret_cast<const uint32_t*>(q_hi + c0 + 8) : 0u;
    }
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const bool first = mod.sink && warp == 0 && split == 0;
    float m_lo = first ? 0.0f : -INFINITY, m_hi = m_lo;
    if (first && sink_logit != nullptr) {            // the heads' learned sink scores, in base 2 like the scores
        m_lo = v_lo ? sink_logit[head0 + h_lo] * kLog2e : 0.0f;
        m_hi = v_hi ? sink_logit[head0 + h_hi] * kLog2e : 0.0f;
    }
    float l_lo = (first && (lane & 3) == 0) ? 1.0f : 0.0f, l_hi = l_lo;

    auto issue = [&](int kt, int stage) {
        const uint32_t ks = smem_u32(pf_smem + (size_t)stage * (kKBytes + kVBytes));
        const uint32_t vs = ks + kKBytes;
        constexpr int kMC = DKP / 8, kKC = MAPS * kMC, kVC = DVP / 8;       // 16-byte pieces of a map's key, a row of keys, a value
        for (int row = threadIdx.x / kKC, chunk = threadIdx.x % kKC; row < kPfN; row += kPfWarps * 32 / kKC) {
            const int key = kt * kPfN + row;
            int page_index, place;
            page_of(key, page_size, page_shift, page_index, place);
            const int page = (key <= pos && key >= lo) ? table[page_index] : -1;
            const bool ok = page >= 0;
            const long long page_at = ok ? (long long)page * page_stride : 0;
            const long long in_page = (long long)g * page_size + place;
            const int in_key = (chunk % kMC) * 8;                       // within its map's key
            const bool k_ok = ok && in_key < dk;
            cp_async_16(ks + (row * kKRow + chunk * 8) * 2, k_plane + (k_ok ? page_at + in_page * kd + (chunk / kMC) * dk + in_key : 0), k_ok);
            if (kKC == kVC) {
                const bool v_ok = ok && chunk * 8 < dv;
                cp_async_16(vs + (row * kVRow + chunk * 8) * 2, v_plane + (v_ok ? page_at + in_page * v_row + chunk * 8 : 0), v_ok);
            }
        }
        if (kKC != kVC) {
            for (int row = threadIdx.x / kVC, chunk = threadIdx.x % kVC; row < kPfN; row += kPfWarps * 32 / kVC) {
                const int key = kt * kPfN + row;
                int page_index, place;
                page_of(key, page_size, page_shift, page_index, place);
                const int page = (key <= pos && key >= lo) ? table[page_index] : -1;
                const bool v_ok = page >= 0 && chunk * 8 < dv;
                cp_async_16(vs + (row * kVRow + chunk * 8) * 2, v_plane + (v_ok ? (long long)page * page_stride + ((long long)g * page_size + place) * v_row + chunk * 8 : 0), v_ok);
            }
        }
        cp_async_commit();
    };

    if (kt_first <= kt_last) issue(kt_first, 0);
    for (int kt = kt_first; kt <= kt_last; ++kt) {
        const int stage = (kt - kt_first) & 1;
        if (kt + 1 <= kt_last) {
            issue(kt + 1, stage ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int key0 = kt * kPfN + warp * 16;                          // this warp's 16 keys of the tile
        if (key0 <= pos && key0 + 15 >= lo) {
            const uint32_t ks_base = smem_u32(pf_smem + (size_t)stage * (kKBytes + kVBytes));
            const uint32_t vs_base = ks_base + kKBytes;
            const int mid = lane >> 3, mrow = lane & 7;
            float s[2][4];
            s[0][0] = s[0][1] = s[0][2] = s[0][3] = s[1][0] = s[1][1] = s[1][2] = s[1][3] = 0.0f;
#pragma unroll
            for (int ks = 0; ks < MAPS * DKP / 16; ++ks) {
                uint32_t kb[4];
                ldmatrix_x4(kb, ks_base + ((warp * 16 + (mid >> 1) * 8 + mrow) * kKRow + ks * 16 + (mid & 1) * 8) * 2);
                const uint32_t b0[2] = {kb[0], kb[1]}, b1[2] = {kb[2], kb[3]};
                mma_bf16_16816(s[0], qa[ks], b0);
                mma_bf16_16816(s[1], qa[ks], b1);
            }
            const int key_base = key0 + (lane & 3) * 2;
            const float d0 = (float)(pos - key_base);
            float tmax_lo = -INFINITY, tmax_hi = -INFINITY;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = key_base + nt * 8 + e;
                    const bool seen = j <= pos && j >= lo;
                    const float dist = d0 - (float)(nt * 8 + e);
                    float a = mod_score_fast(s[nt][e], slope_lo, dist, mod, inv_cap);
                    float b = mod_score_fast(s[nt][2 + e], slope_hi, dist, mod, inv_cap);
                    if (mod.dist_bias != nullptr) {
                        a += dist_bias_of(mod, head0 + (v_lo ? h_lo : 0), pos - j) * kLog2e;
                        b += dist_bias_of(mod, head0 + (v_hi ? h_hi : 0), pos - j) * kLog2e;
                    }
                    s[nt][e] = (seen && v_lo) ? a : -INFINITY;
                    s[nt][2 + e] = (seen && v_hi) ? b : -INFINITY;
                    tmax_lo = fmaxf(tmax_lo, s[nt][e]);
                    tmax_hi = fmaxf(tmax_hi, s[nt][2 + e]);
                }
            tmax_lo = fmaxf(tmax_lo, __shfl_xor_sync(0xffffffffu, tmax_lo, 1));
            tmax_lo = fmaxf(tmax_lo, __shfl_xor_sync(0xffffffffu, tmax_lo, 2));
            tmax_hi = fmaxf(tmax_hi, __shfl_xor_sync(0xffffffffu, tmax_hi, 1));
            tmax_hi = fmaxf(tmax_hi, __shfl_xor_sync(0xffffffffu, tmax_hi, 2));
            const float mn_lo = fmaxf(m_lo, tmax_lo), mn_hi = fmaxf(m_hi, tmax_hi);
            const float ms_lo = mn_lo == -INFINITY ? 0.0f : mn_lo, ms_hi = mn_hi == -INFINITY ? 0.0f : mn_hi;
            const float c_lo = fast_exp2(m_lo - ms_lo), c_hi = fast_exp2(m_hi - ms_hi);
            m_lo = mn_lo;
            m_hi = mn_hi;
            float sum_lo = 0.0f, sum_hi = 0.0f;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    s[nt][e] = fast_exp2(s[nt][e] - ms_lo);
                    s[nt][2 + e] = fast_exp2(s[nt][2 + e] - ms_hi);
                    sum_lo += s[nt][e];
                    sum_hi += s[nt][2 + e];
                }
            l_lo = l_lo * c_lo + sum_lo;
            l_hi = l_hi * c_hi + sum_hi;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) {
                o[i][0] *= c_lo; o[i][1] *= c_lo; o[i][2] *= c_hi; o[i][3] *= c_hi;
            }
            const uint32_t pa[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]),
                                    pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
            for (int c = 0; c < DVP / 8; c += 2) {
                uint32_t vb[4];
                ldmatrix_x4_trans(vb, vs_base + ((warp * 16 + (mid & 1) * 8 + mrow) * kVRow + (c + (mid >> 1)) * 8) * 2);
                const uint32_t b0[2] = {vb[0], vb[1]}, b1[2] = {vb[2], vb[3]};
                mma_bf16_16816(o[c], pa, b0);
                mma_bf16_16816(o[c + 1], pa, b1);
            }
        }
        __syncthreads();
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    // the warps meet: [warp][row of the tile in use][dv + 2] floats, over the staging buffers (all reads of which are done)
    float* meet = reinterpret_cast<float*>(pf_smem);
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) {
        const int col = i * 8 + (lane & 3) * 2;
        if (col >= dv) continue;
        if (v_lo) { float* d = meet + ((size_t)warp * used + r_lo) * rec; d[col] = o[i][0]; d[col + 1] = o[i][1]; }
        if (v_hi) { float* d = meet + ((size_t)warp * used + r_hi) * rec; d[col] = o[i][2]; d[col + 1] = o[i][3]; }
    }
    if ((lane & 3) == 0) {
        if (v_lo) { float* d = meet + ((size_t)warp * used + r_lo) * rec; d[dv] = m_lo; d[dv + 1] = l_lo; }
        if (v_hi) { float* d = meet + ((size_t)warp * used + r_hi) * rec; d[dv] = m_hi; d[dv + 1] = l_hi; }
    }
    __syncthreads();
    // element e of row h of the tile, added over the warps: its sum, the weights' sum and their maximum (base 2)
    auto add_warps = [&](int h, int e, float& v, float& total, float& mm) {
        mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < kPfWarps; ++w) mm = fmaxf(mm, meet[((size_t)w * used + h) * rec + dv]);
        total = v = 0.0f;
#pragma unroll
        for (int w = 0; w < kPfWarps; ++w) {
            const float* src = meet + ((size_t)w * used + h) * rec;
            const float wt = src[dv] == -INFINITY ? 0.0f : fast_exp2(src[dv] - mm);
            total += src[dv + 1] * wt;
            v += src[e] * wt;
        }
    };
    if (MAPS > 1 && splits == 1) {                    // a warp per head: the difference of its two rows, normed
        for (int h = warp; h < group; h += kPfWarps) {
            float d[DVP / 32], sum = 0.0f;
#pragma unroll
            for (int c = 0; c < DVP / 32; ++c) {
                const int e = lane + 32 * c;
                d[c] = 0.0f;
                if (e < dv) {
                    float v1, v2, t1, t2, mm;
                    add_warps(h, e, v1, t1, mm);
                    add_warps(group + h, e, v2, t2, mm);
                    d[c] = (t1 > 0.0f ? v1 / t1 : 0.0f) - diff.lambda * (t2 > 0.0f ? v2 / t2 : 0.0f);
                }
                sum += d[c] * d[c];
            }
            const float norm = diff.out_scale / sqrtf(warp_sum(sum) / (float)dv + diff.eps);
#pragma unroll
            for (int c = 0; c < DVP / 32; ++c) {
                const int e = lane + 32 * c;
                if (e >= dv) continue;
                float v = d[c] * norm;
                if (gate != nullptr)
                    v *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)t * gate_stride + gate_at(mod.gate_per_head, head0 + h, dv, e)])));
                out[((size_t)t * q_heads + head0 + h) * dv + e] = __float2bfloat16_rn(v);
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < used * dv; i += blockDim.x) {
        const int h = i / dv, e = i % dv;
        float mm, total, v;
        add_warps(h, e, v, total, mm);
        if (splits > 1) {
            // [row of the grid][head (, map)][split][dv + 2]: sums, then maximum (base 2) and weight
            const int map = MAPS > 1 && h >= group ? 1 : 0;
            float* dst = part + ((((size_t)blockIdx.x * q_heads + head0 + h - map * group) * MAPS + map) * splits + split) * rec;
            dst[e] = v;
            if (e == 0) { dst[dv] = mm; dst[dv + 1] = total; }
            continue;
        }
        v = total > 0.0f ? v / total : 0.0f;
        if (gate != nullptr)
            v *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)t * gate_stride + gate_at(mod.gate_per_head, head0 + h, dv, e)])));
        out[((size_t)t * q_heads + head0 + h) * dv + e] = __float2bfloat16_rn(v);
    }
}

// The runs of a (row, head) added in their order (with two maps: of both, then the normed difference), the gate
// applied, the result written.
template <int MAPS>
__global__ void attention_biased_combine_kernel(const float* part, const int* __restrict__ token_slot,
                                                const int* __restrict__ rows, int q_heads, int dv, int splits,
                                                const bf16* gate, int gate_stride, int gate_per_head, DiffMod diff,
                                                bf16* __restrict__ out) {
    __shared__ float scratch[32], row_s[MAPS > 1 ? 128 : 1];
    TLLM_PDL_ENTER();
    const int t = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
    const int head = blockIdx.y, rec = dv + 2;
    bf16* dst = out + ((size_t)t * q_heads + head) * dv;
    if (token_slot[t] < 0) {
        for (int e = threadIdx.x; e < dv; e += blockDim.x) dst[e] = __float2bfloat16_rn(0.0f);
        return;
    }
    float norm = 1.0f, mm[MAPS];
    const float* src[MAPS];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        src[mp] = part + (((size_t)blockIdx.x * q_heads + head) * MAPS + mp) * splits * rec;
        mm[mp] = -INFINITY;
        for (int s2 = 0; s2 < splits; ++s2) mm[mp] = fmaxf(mm[mp], src[mp][s2 * rec + dv]);
    }
    auto added = [&](int mp, int e) -> float {
        float total = 0.0f, v = 0.0f;
        for (int s2 = 0; s2 < splits; ++s2) {
            const float ms = src[mp][s2 * rec + dv];
            const float w = ms == -INFINITY ? 0.0f : fast_exp2(ms - mm[mp]);
            total += src[mp][s2 * rec + dv + 1] * w;
            v += src[mp][s2 * rec + e] * w;
        }
        return total > 0.0f ? v / total : 0.0f;
    };
    if (MAPS > 1) {
        float sum = 0.0f;
        for (int e = threadIdx.x; e < dv; e += blockDim.x) {
            const float v = added(0, e) - diff.lambda * added(MAPS - 1, e);
            row_s[e] = v;                             // only this thread looks at element e
            sum += v * v;
        }
        norm = diff.out_scale / sqrtf(block_sum(sum, scratch) / (float)dv + diff.eps);
    }
    for (int e = threadIdx.x; e < dv; e += blockDim.x) {
        float v = MAPS > 1 ? row_s[e] * norm : added(0, e);
        if (gate != nullptr) v *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)t * gate_stride + gate_at(gate_per_head, head, dv, e)])));
        dst[e] = __float2bfloat16_rn(v);
    }
}

// Blocks that share a key/value head's query heads in the one-token kernel: the fewest that leave each at
// most the tile's 16 rows (`maps` of them per head) and divide the heads evenly; 0 if there is no such number.
static int biased_sub_groups(int group, int maps) {
    for (int s = 1; s <= group; ++s)
        if (group % s == 0 && group / s * maps <= 16) return s;
    return 0;
}

template <int DKP, int DVP, int MAPS>
static int launch_biased_decode(const void* q, const void* kp, const void* vp, long long page_stride,
                                const int* positions, const int* token_slot, const int* rows, int n_rows,
                                const int* block_table, int max_pages, int page_size, int q_heads, int kv_heads,
                                int dk, int dv, ScoreMod mod, DiffMod diff, const float* slopes, const float* sink_logit, int v_row,
                                const void* gate, int gate_stride, int splits, float* part, void* out, cudaStream_t stream) {
    const size_t smem = (size_t)2 * kPfN * ((MAPS * DKP + kPfPad) + (DVP + kPfPad)) * 2;      // also holds the warps' meeting
    static OncePerDevice configured;
    if (configured.first()) {
        cudaError_t e = cudaFuncSetAttribute(attention_biased_decode_kernel<DKP, DVP, MAPS>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { set_error("attention_biased_decode: %s", cudaGetErrorString(e)); return (int)e; }
        configured.done();
    }
    const int sub_groups = biased_sub_groups(q_heads / kv_heads, MAPS);
    launch_pdl(kPdlAttention, attention_biased_decode_kernel<DKP, DVP, MAPS>, dim3(n_rows, kv_heads * sub_groups, splits), dim3(kPfWarps * 32),
               smem, stream, (const bf16*)q, (const bf16*)kp, (const bf16*)vp, page_stride, positions, token_slot,
               rows, block_table, max_pages, page_size, page_shift_of(page_size), q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row,
               (const bf16*)gate, gate_stride, splits, sub_groups, part, (bf16*)out);
    if (splits > 1)
        launch_pdl(kPdlCombine, attention_biased_combine_kernel<MAPS>, dim3(n_rows, q_heads), dim3(dv >= 128 ? 128 : 64), 0, stream,
                   (const float*)part, token_slot, rows, q_heads, dv, splits, (const bf16*)gate, gate_stride, mod.gate_per_head, diff, (bf16*)out);
    return finish_launch("attention_biased_decode");
}

}  // namespace tllm

using namespace tllm;

extern "C" {

int tllm_qkv_unit_store(const void* proj, int row_stride, const void* q_gain, const void* k_gain, float eps,
                        int do_norm, const int* positions, const int* token_slot, const int* block_table,
                        int max_pages, int page_size, void* k_plane, void* v_plane, long long page_stride,
                        void* q_out, int dtype, int tokens, int q_heads, int kv_heads, int dk, int dv,
                        int store, const float* inv_freq, int rot_dims, int rot_pairs, float temp_coef, int temp_every,
                        int v_from_k, const float* bias, const void* mix_first, int mix_stride, const float* mix_bias,
                        float mix_share, cudaStream_t stream) {
    TLLM_REQUIRE(tokens >= 0 && q_heads > 0 && kv_heads > 0 && dk > 0 && dv > 0, "qkv_unit_store: bad sizes");
    TLLM_REQUIRE(row_stride >= (q_heads + kv_heads) * dk + (v_from_k ? 0 : kv_heads * dv), "qkv_unit_store: rows of %d are too short", row_stride);
    TLLM_REQUIRE(rot_dims >= 0 && rot_dims <= dk && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq != nullptr),
                 "qkv_unit_store: a rotation of %d of %d elements", rot_dims, dk);
    TLLM_REQUIRE(!v_from_k || dv == dk, "qkv_unit_store: keys of width %d cannot serve as values of width %d", dk, dv);
    TLLM_REQUIRE(temp_every >= 0, "qkv_unit_store: negative constant");
    TLLM_REQUIRE(do_norm >= kQkNone && do_norm <= kQkWhole, "qkv_unit_store: unknown norm %d", do_norm);
    TLLM_REQUIRE(!do_norm || eps > 0.0f, "qkv_unit_store: eps must be positive");
    TLLM_REQUIRE(mix_first == nullptr || (!v_from_k && mix_stride >= kv_heads * dv), "qkv_unit_store: other values in rows of %d", mix_stride);
    TLLM_REQUIRE(!store || (k_plane && v_plane && block_table && page_size > 0 && max_pages > 0),
                 "qkv_unit_store: no cache to write to");
    TLLM_REQUIRE(q_out != nullptr, "qkv_unit_store: no place for the queries");
    if (tokens == 0) return 0;
    const int heads = q_heads + 2 * kv_heads;
    const int warps = heads >= 8 ? 8 : (heads >= 4 ? 4 : 2);
#define STORE(T)                                                                                              \
    launch_pdl(kPdlQk, qkv_unit_store_kernel<T>, dim3(tokens), dim3(warps * 32), 0, stream, (const T*)proj,   \
               row_stride, (const T*)q_gain, (const T*)k_gain, eps, do_norm, positions, token_slot,           \
               block_table, max_pages, page_size, (T*)k_plane, (T*)v_plane, page_stride, (T*)q_out, q_heads,  \
               kv_heads, dk, dv, store, inv_freq, rot_dims, rot_pairs, temp_coef, temp_every, v_from_k, bias, \
               ValueMix<T>{(const T*)mix_first, mix_stride, mix_bias, 1.0f - mix_share, mix_share})
    auto aligned16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
    const bool vec = dtype == kBF16 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && (rot_pairs || rot_dims % 16 == 0) &&
                     row_stride % 8 == 0 && page_stride % 8 == 0 && aligned16(proj) && aligned16(q_out) &&
                     aligned16(k_plane) && aligned16(v_plane) && aligned16(q_gain) && aligned16(k_gain) && aligned16(bias) &&
                     (mix_first == nullptr || (aligned16(mix_first) && mix_stride % 8 == 0));
    const int sms = sm_count_cached() > 0 ? sm_count_cached() : 148;
    auto split_of = [&](int per_warp) {               // blocks per token: up to one run of heads per warp
        int split = 1;
        while (split * 8 * per_warp < q_heads + kv_heads && (long long)tokens * (split + 1) <= 2LL * sms) ++split;
        return split;
    };
#define STORE_VEC(GS)                                                                                             \
    launch_pdl(kPdlQk, qkv_unit_store_vec_kernel<GS>, dim3(tokens, split_of(32 / GS)), dim3(256), (size_t)rot_dims * sizeof(float),  \
               stream, (const bf16*)proj, row_stride, (const bf16*)q_gain, (const bf16*)k_gain, eps, do_norm,     \
               positions, token_slot, block_table, max_pages, page_size, (bf16*)k_plane, (bf16*)v_plane,          \
               page_stride, (bf16*)q_out, q_heads, kv_heads, dk, dv, store, inv_freq, rot_dims, rot_pairs, temp_coef, \
               temp_every, v_from_k, bias, ValueMix<bf16>{(const bf16*)mix_first, mix_stride, mix_bias, 1.0f - mix_share, mix_share})
    if (vec) {
        if (dk <= 8) STORE_VEC(1);
        else if (dk <= 16) STORE_VEC(2);
        else if (dk <= 32) STORE_VEC(4);
        else if (dk <= 64) STORE_VEC(8);
        else if (dk <= 128) STORE_VEC(16);
        else STORE_VEC(32);
    } else if (dtype == kBF16) STORE(bf16);
    else if (dtype == kF32) STORE(float);
    else TLLM_REQUIRE(false, "qkv_unit_store: unknown dtype %d", dtype);
#undef STORE
#undef STORE_VEC
    return finish_launch("qkv_unit_store");
}

int tllm_attention_biased_general(
    const void* q, const void* k_plane, const void* v_plane, long long page_stride, const int* positions,
    const int* token_slot, const int* block_table, int max_pages, int page_size, int dtype, int tokens,
    int q_heads, int kv_heads, int dk, int dv, float scale, float softcap, int chunk, int window, int sink,
    const float* slopes, const float* sink_logit, const float* dist_bias, int dist_len, int v_row, const void* gate, int gate_stride, int gate_per_head,
    int maps, float lambda, float diff_eps, float diff_scale, void* out, cudaStream_t stream) {
    if (v_row <= 0) v_row = dv;
    TLLM_REQUIRE(maps == 1 || (maps == 2 && diff_eps > 0.0f), "attention_biased: %d maps", maps);
    const DiffMod diff{lambda, diff_eps, diff_scale};
    TLLM_REQUIRE(dist_bias == nullptr || dist_len > 0, "attention_biased: an empty table of biases");
    TLLM_REQUIRE(v_row >= dv, "attention_biased: values of width %d in rows of %d", dv, v_row);
    TLLM_REQUIRE(tokens >= 0 && q_heads > 0 && kv_heads > 0 && q_heads % kv_heads == 0,
                 "attention_biased: %d query heads over %d key/value heads", q_heads, kv_heads);
    TLLM_REQUIRE(dk > 0 && dk <= 512 && dv > 0 && dv <= 512, "attention_biased: widths %d, %d outside 1..512", dk, dv);
    TLLM_REQUIRE(page_size > 0 && max_pages > 0, "attention_biased: bad page geometry");
    TLLM_REQUIRE(tokens <= 65535, "attention_biased: %d tokens in one step exceed 65535", tokens);
    TLLM_REQUIRE(chunk >= 0 && window >= 0 && softcap >= 0.0f, "attention_biased: negative constant");
    if (tokens == 0) return 0;
    const ScoreMod mod{scale, softcap, chunk, window, sink ? 1 : 0, dist_bias, dist_len, gate_per_head ? 1 : 0};
#define GEN(T, M) launch_general<T, M>(q, k_plane, v_plane, page_stride, positions, token_slot, block_table, max_pages, page_size, \
                                       tokens, q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row, gate, gate_stride, out, stream)
    if (dtype == kBF16) return maps == 2 ? GEN(bf16, 2) : GEN(bf16, 1);
    if (dtype == kF32) return maps == 2 ? GEN(float, 2) : GEN(float, 1);
#undef GEN
    TLLM_REQUIRE(false, "attention_biased: unknown dtype %d", dtype);
}

// Whether the two bfloat16 kernels below take these sizes (else the general kernel serves).  dk: width of one map's key.
int tllm_attention_maps_fast_ok(int q_heads, int kv_heads, int dk, int dv, int maps) {
    return q_heads > 0 && kv_heads > 0 && q_heads % kv_heads == 0 && biased_sub_groups(q_heads / kv_heads, maps) > 0 &&
           kv_heads * biased_sub_groups(q_heads / kv_heads, maps) <= 65535 &&
           dk % 8 == 0 && dv % 8 == 0 && dk > 0 && dv > 0 && dk <= 128 && dv <= 128;
}
int tllm_attention_biased_fast_ok(int q_heads, int kv_heads, int dk, int dv) {
    return tllm_attention_maps_fast_ok(q_heads, kv_heads, dk, dv, 1);
}

// seg_info: int[segments][4] = slot, first row, length, position of the first row.
// tiles: int[n_tiles][2] = segment, offset of the block's first query row in the segment.
int tllm_attention_biased_prefill(
    const void* q, const void* k_plane, const void* v_plane, long long page_stride, const int* seg_info,
    const int* tiles, int n_tiles, const int* block_table, int max_pages, int page_size, int q_heads,
    int kv_heads, int dk, int dv, float scale, float softcap, int chunk, int window, int sink,
    const float* slopes, const float* sink_logit, const float* dist_bias, int dist_len, int v_row, const void* gate, int gate_stride, int gate_per_head,
    int maps, float lambda, float diff_eps, float diff_scale, void* out, cudaStream_t stream) {
    if (v_row <= 0) v_row = dv;
    TLLM_REQUIRE(maps == 1 || (maps == 2 && diff_eps > 0.0f), "attention_biased_prefill: %d maps", maps);
    const DiffMod diff{lambda, diff_eps, diff_scale};
    TLLM_REQUIRE(dist_bias == nullptr || dist_len > 0, "attention_biased_prefill: an empty table of biases");
    TLLM_REQUIRE(v_row >= dv && v_row % 8 == 0, "attention_biased_prefill: values of width %d in rows of %d", dv, v_row);
    TLLM_REQUIRE(tllm_attention_maps_fast_ok(q_heads, kv_heads, dk, dv, maps), "attention_biased_prefill: sizes %d/%d heads, widths %d/%d", q_heads, kv_heads, dk, dv);
    TLLM_REQUIRE(page_size > 0 && max_pages > 0 && n_tiles >= 0 && q_heads <= 65535, "attention_biased_prefill: bad geometry");
    TLLM_REQUIRE(chunk >= 0 && window >= 0 && softcap >= 0.0f, "attention_biased_prefill: negative constant");
    TLLM_REQUIRE(gate == nullptr || gate_per_head || gate_stride % 2 == 0, "attention_biased_prefill: odd gate stride");
    if (n_tiles == 0) return 0;
    const ScoreMod mod{scale, softcap, chunk, window, sink ? 1 : 0, dist_bias, dist_len, gate_per_head ? 1 : 0};
#define PF_M(A, B, M) launch_biased_prefill<A, B, M>(q, k_plane, v_plane, page_stride, seg_info, tiles, n_tiles, block_table, max_pages, \
                                             page_size, q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row, gate, gate_stride, out, stream)
#define PF(A, B) (maps == 2 ? PF_M(A, B, 2) : PF_M(A, B, 1))
    if (dk <= 64) return dv <= 64 ? PF(64, 64) : PF(64, 128);
    return dv <= 64 ? PF(128, 64) : PF(128, 128);
#undef PF
#undef PF_M
}

// rows: indices of the one-token rows (null: rows 0 .. n_rows - 1).  splits: runs of keys per (row,
// key/value head), each a block; with more than one, `part` holds n_rows * q_heads * maps * splits * (dv + 2) floats.
int tllm_attention_biased_decode(
    const void* q, const void* k_plane, const void* v_plane, long long page_stride, const int* positions,
    const int* token_slot, const int* rows, int n_rows, const int* block_table, int max_pages, int page_size,
    int q_heads, int kv_heads, int dk, int dv, float scale, float softcap, int chunk, int window, int sink,
    const float* slopes, const float* sink_logit, const float* dist_bias, int dist_len, int v_row, const void* gate,
    int gate_stride, int gate_per_head, int maps, float lambda, float diff_eps, float diff_scale, int splits, float* part,
    void* out, cudaStream_t stream) {
    if (v_row <= 0) v_row = dv;
    TLLM_REQUIRE(maps == 1 || (maps == 2 && diff_eps > 0.0f), "attention_biased_decode: %d maps", maps);
    const DiffMod diff{lambda, diff_eps, diff_scale};
    TLLM_REQUIRE(dist_bias == nullptr || dist_len > 0, "attention_biased_decode: an empty table of biases");
    TLLM_REQUIRE(v_row >= dv && v_row % 8 == 0, "attention_biased_decode: values of width %d in rows of %d", dv, v_row);
    TLLM_REQUIRE(tllm_attention_maps_fast_ok(q_heads, kv_heads, dk, dv, maps), "attention_biased_decode: sizes %d/%d heads, widths %d/%d", q_heads, kv_heads, dk, dv);
    TLLM_REQUIRE(page_size > 0 && max_pages > 0 && n_rows >= 0 && kv_heads <= 65535, "attention_biased_decode: bad geometry");
    TLLM_REQUIRE(chunk >= 0 && window >= 0 && softcap >= 0.0f, "attention_biased_decode: negative constant");
    TLLM_REQUIRE(splits >= 1 && splits <= 64 && (splits == 1 || part != nullptr), "attention_biased_decode: %d runs of keys", splits);
    if (n_rows == 0) return 0;
    const ScoreMod mod{scale, softcap, chunk, window, sink ? 1 : 0, dist_bias, dist_len, gate_per_head ? 1 : 0};
#define DEC_M(A, B, M) launch_biased_decode<A, B, M>(q, k_plane, v_plane, page_stride, positions, token_slot, rows, n_rows, block_table, \
                                             max_pages, page_size, q_heads, kv_heads, dk, dv, mod, diff, slopes, sink_logit, v_row, gate, gate_stride, \
                                             splits, part, out, stream)
#define DEC(A, B) (maps == 2 ? DEC_M(A, B, 2) : DEC_M(A, B, 1))
    if (dk <= 64) return dv <= 64 ? DEC(64, 64) : DEC(64, 128);
    return dv <= 64 ? DEC(128, 64) : DEC(128, 128);
#undef DEC
#undef DEC_M
}

}  // extern "C"
