// Per-head RMSNorm + rotary encoding + cache write, and attention over the cache
// for any element type, head size and number of heads.
//
// Formulas (reference):
//  * fused per-head norm and rotation, norm before rotation, half-split pairing:
//      n_c = x_c * (1/sqrt(sum(x^2)/d + eps)) * w_c
//      out_c = n_c * cos[pos, c mod half] + r_c * sin[pos, c mod half],
//      r_c = -n_{c+half} for c < half, n_{c-half} otherwise
//    (src/kidi/layers/qwen3.cpp:37-48, src/kidi/ops/context.cpp:1051-1065,
//     src/kidi/runtime/mps/eager_kernels.metal:87-97)
//  * scores s = (q . k) * scale, key head = query head / (heads / kv_heads), softmax
//    over the visible keys, output = sum p_u v_u
//    (src/kidi/layers/qwen3.cpp:53-54, src/kidi/runtime/vulkan/attention.comp:32-101)
//  * the causal rule is the generic causal path's: key u is visible to the query at
//    position p when u <= p (src/kidi/model/gemma4.cpp:736-740); with a window W,
//    when also u > p - W; with chunks of C positions, when also floor(u / C) = floor(p / C).
//  * instead of the softmax a key's weight can be sigmoid(s + b_h), b_h a number per head, normalised over nothing.
//  * a number from a table [heads, distance] can be added to a score (p - u is the distance), and a value can be the key as
//    it was before its norm: then only that is kept, s = r_u (q . k_u) scale with r_u = 1 / sqrt(sum(k_u^2)/d + eps), and the
//    norm's weight rides in q.
// Norm sums, rotation, scores, softmax and the weighted sum are 32-bit.
#include "common.cuh"

struct RopeStoreArgs {
    void* qkv;                 // [rows, ld] : q heads, then k heads, then v heads, each head_dim wide
    long long ld;
    const void* q_norm;        // [head_dim] or null
    const void* k_norm;        // [head_dim] or null
    const float* cos_table;    // [positions, rotary_dim/2] or null (no rotation)
    const float* sin_table;
    const int* row_seq;        // [rows]  (-1: padding row, skipped)
    const int* row_pos;        // [rows]
    const int* seq_slot;       // [seqs]
    const int* seq_start;      // [seqs]
    const int* seq_len;        // [seqs]
    void* k_cache;             // storage of this schedule entry, or null (no write)
    void* v_cache;
    CacheGeometry cache;
    int rows, heads, kv_heads, head_dim, rotary_dim;
    float eps;
    int transform;             // 0: only copy the k and v heads, as they are, to the cache
    int value_dim;             // width of a v head (0: head_dim); the v heads follow the k heads in a row
    const float* q_scale;      // [positions] or null: a q head at position p is multiplied by q_scale[p] (after the
                               // norm and the rotation)
    int tied;                  // values are the keys before their norm: a row holds q heads and k heads, the k heads stay as
                               // they are and are what the cache keeps (k_cache)
    void* k_normed;            // [rows, ld_k_normed] or null (tied): takes the k heads divided by their root mean squares
    long long ld_k_normed;
};

// One warp per (row, head) over heads + 2*kv_heads heads (heads + kv_heads where values are keys).
template <typename T, typename TW>
__global__ void __launch_bounds__(128) rope_store_kernel(RopeStoreArgs a) {
    __shared__ float normed[4][256];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first_head = a.transform ? 0 : a.heads;         // copying alone: the k (and v) heads only
    const int total_heads = a.heads - first_head + (a.tied ? 1 : 2) * a.kv_heads;
    const long long item = (long long)blockIdx.x * 4 + warp;
    if (item >= (long long)a.rows * total_heads) return;
    const int row = (int)(item / total_heads);
    const int head = first_head + (int)(item - (long long)row * total_heads);
    const int seq = a.row_seq[row];
    if (seq < 0) return;
    const int position = a.row_pos[row];
    const int d = a.head_dim;
    const int vd = a.value_dim ? a.value_dim : d;
    const bool is_value = head >= a.heads + a.kv_heads;
    T* vector = (T*)a.qkv + row * a.ld +
                (is_value ? (long long)(a.heads + a.kv_heads) * d + (long long)(head - a.heads - a.kv_heads) * vd
                          : (long long)head * d);

    // Where this head goes in the cache, if anywhere.
    T* cached = nullptr;
    if (head >= a.heads && a.k_cache) {
        bool keep = true;
        if (a.cache.ring_pages) {  // a ring keeps the last ring_tokens tokens of the step only
            const int ring_tokens = a.cache.ring_pages << a.cache.page_shift;
            keep = position >= a.seq_start[seq] + a.seq_len[seq] - ring_tokens;
        }
        if (keep) {
            const int kv_head = is_value ? head - a.heads - a.kv_heads : head - a.heads;
            const long long offset = cache_row_offset(a.cache, a.seq_slot[seq], position, kv_head);
            cached = is_value ? (T*)a.v_cache + offset / d * vd : (T*)a.k_cache + offset;
        }
    }

    const bool raw_key = a.tied && head >= a.heads;
    if (is_value || !a.transform || raw_key) {  // a value head, or copy only
        const int width = is_value ? vd : d;
        if (cached)
            for (int c = lane; c < width; c += 32) cached[c] = vector[c];
        if (raw_key && a.transform && a.k_normed) {
            float square = 0.f;
            for (int c = lane; c < d; c += 32) square = fmaf(to_float(vector[c]), to_float(vector[c]), square);
            const float inv = 1.0f / sqrtf(warp_sum(square) / (float)d + a.eps);
            T* normed_key = (T*)a.k_normed + row * a.ld_k_normed + (long long)(head - a.heads) * d;
            for (int c = lane; c < d; c += 32) normed_key[c] = from_float<T>(to_float(vector[c]) * inv);
        }
        return;
    }

    const TW* weight = (const TW*)(head < a.heads ? a.q_norm : a.k_norm);
    float values[8];
    float square = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        values[i] = c < d ? to_float(vector[c]) : 0.f;
        square = fmaf(values[i], values[i], square);
    }
    float inv = 1.f;
    if (weight) inv = 1.0f / sqrtf(warp_sum(square) / (float)d + a.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < d) {
            if (weight) values[i] = values[i] * inv * to_float(weight[c]);
            normed[warp][c] = values[i];
        }
    }
    __syncwarp();
    const int half = a.rotary_dim / 2;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c >= d) continue;
        float out = values[i];
        if (a.cos_table && c < a.rotary_dim) {
            const int j = c < half ? c : c - half;
            const float cosine = a.cos_table[(long long)position * half + j];
            const float sine = a.sin_table[(long long)position * half + j];
            const float rotated = c < half ? -normed[warp][c + half] : normed[warp][c - half];
            out = values[i] * cosine + rotated * sine;
        }
        if (a.q_scale && head < a.heads) out *= a.q_scale[position];
        const T stored = from_float<T>(out);
        vector[c] = stored;
        if (cached) cached[c] = stored;
    }
}

// Eight consecutive norm weights as 32-bit values (the address is 16-byte aligned: the head
// width is a multiple of eight).
__device__ __forceinline__ void load8(const float* p, float (&w)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
}
__device__ __forceinline__ void load8(const bf16* p, float (&w)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 two = __bfloat1622float2(pairs[i]);
        w[2 * i] = two.x;
        w[2 * i + 1] = two.y;
    }
}

// The same for bfloat16 rows in 16-byte vectors. A (row, head) is handled by a group of
// L lanes (L the power of two that covers head_dim / 8: 16 lanes for a head of 128), so a
// warp takes 32 / L of them; lane l of a group owns elements 8l..8l+7 of the head, and its
// rotation partners are the eight elements of lane l +- half/8, fetched with shuffles.
// Needs head_dim and rotary_dim/2 to be multiples of 8 and 16-byte aligned rows.
template <typename TW>
__global__ void __launch_bounds__(128) rope_store_bf16_kernel(RopeStoreArgs a, int group_lanes) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first_head = a.transform ? 0 : a.heads;         // copying alone: the k (and v) heads only
    const int total_heads = a.heads - first_head + (a.tied ? 1 : 2) * a.kv_heads;
    const int per_warp = 32 / group_lanes;
    const int group = lane / group_lanes, l = lane - group * group_lanes;
    const int item = (blockIdx.x * 4 + warp) * per_warp + group;   // the launcher keeps the count below 2^31
    // Every lane stays to the end (the shuffles are warp-wide); `alive` says whether the
    // group has a (row, head) to work on.
    bool alive = item < a.rows * total_heads;
    const int row = alive ? item / total_heads : 0;
    const int head = alive ? first_head + item - row * total_heads : first_head;
    const int d = a.head_dim, c0 = 8 * l;
    bf16* vector = (bf16*)a.qkv + (long long)row * a.ld + head * d;
    // The row's elements are asked for together with its sequence and position (a padding
    // row's elements are there to be read; nothing of it is stored).
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    if (alive && c0 < d) raw = *reinterpret_cast<const uint4*>(vector + c0);
    const int seq = a.row_seq[row];
    const int position = a.row_pos[row];
    alive = alive && seq >= 0;
    const bool mine = alive && c0 < d;

    bf16* cached = nullptr;
    if (alive && head >= a.heads && a.k_cache) {
        bool keep = true;
        if (a.cache.ring_pages) {
            const int ring_tokens = a.cache.ring_pages << a.cache.page_shift;
            keep = position >= a.seq_start[seq] + a.seq_len[seq] - ring_tokens;
        }
        if (keep) {
            const bool is_key = head < a.heads + a.kv_heads;
            const int kv_head = is_key ? head - a.heads : head - a.heads - a.kv_heads;
            cached = (bf16*)(is_key ? a.k_cache : a.v_cache) +
                     cache_row_offset(a.cache, a.seq_slot[seq], position, kv_head);
        }
    }
    if (!mine) raw = make_uint4(0u, 0u, 0u, 0u);
    const bool raw_key = a.tied && head >= a.heads;
    const bool plain = head >= a.heads + a.kv_heads || !a.transform || raw_key;  // a value head, or copy only
    if (plain && cached && mine) *reinterpret_cast<uint4*>(cached + c0) = raw;
    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
    float v[8];
    float square = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 two = __bfloat1622float2(pairs[i]);
        v[2 * i] = two.x;
        v[2 * i + 1] = two.y;
        square = fmaf(two.x, two.x, square);
        square = fmaf(two.y, two.y, square);
    }
    const TW* weight = (const TW*)(head < a.heads ? a.q_norm : a.k_norm);
    if (a.q_norm || a.k_norm) {      // the same for the whole launch: the shuffles stay warp-wide
        for (int offset = group_lanes >> 1; offset > 0; offset >>= 1)
            square += __shfl_xor_sync(0xffffffffu, square, offset);
        if (weight && mine && !plain) {
            const float inv = 1.0f / sqrtf(square / (float)d + a.eps);
            float w[8];
            load8(weight + c0, w);
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = v[i] * inv * w[i];
        }
        if (raw_key && a.k_normed && a.transform && mine) {
            const float inv = 1.0f / sqrtf(square / (float)d + a.eps);
            uint4 packed;
            __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
            for (int i = 0; i < 4; ++i) out[i] = __floats2bfloat162_rn(v[2 * i] * inv, v[2 * i + 1] * inv);
            *reinterpret_cast<uint4*>((bf16*)a.k_normed + row * a.ld_k_normed + (head - a.heads) * d + c0) = packed;
        }
    }
    if (a.cos_table) {
        const int half = a.rotary_dim / 2;
        const bool low = c0 < half;
        const int partner = group * group_lanes + ((low ? l + half / 8 : l - half / 8) & (group_lanes - 1));
        float other[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) other[i] = __shfl_sync(0xffffffffu, v[i], partner);
        if (mine && !plain && c0 < a.rotary_dim) {
            const int j = low ? c0 : c0 - half;
            const float4* cosine = reinterpret_cast<const float4*>(a.cos_table + (long long)position * half + j);
            const float4* sine = reinterpret_cast<const float4*>(a.sin_table + (long long)position * half + j);
            const float4 ca = cosine[0], cb = cosine[1], sa = sine[0], sb = sine[1];
            const float c8[8] = {ca.x, ca.y, ca.z, ca.w, cb.x, cb.y, cb.z, cb.w};
            const float s8[8] = {sa.x, sa.y, sa.z, sa.w, sb.x, sb.y, sb.z, sb.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = v[i] * c8[i] + (low ? -other[i] : other[i]) * s8[i];
        }
    }
    if (mine && !plain && a.q_scale && head < a.heads) {
        const float factor = a.q_scale[position];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= factor;
    }
    if (mine && !plain) {
        uint4 packed;
        __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
        for (int i = 0; i < 4; ++i) out[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(vector + c0) = packed;
        if (cached) *reinterpret_cast<uint4*>(cached + c0) = packed;
    }
}

KIDI_API int kidi_rope_store(const RopeStoreArgs* args, int dtype, int norm_dtype, cudaStream_t stream) {
    const RopeStoreArgs& a = *args;
    if (a.rows <= 0) return 0;
    if (a.head_dim > 256 || a.head_dim <= 0 || a.rotary_dim > a.head_dim || (a.rotary_dim & 1) || a.value_dim < 0)
        return KIDI_REFUSED_SIZE;
    if (a.tied && (a.cos_table || a.v_cache || !a.q_norm || (a.value_dim && a.value_dim != a.head_dim)) && a.transform)
        return KIDI_REFUSED_SIZE;
    const long long items = (long long)a.rows * ((a.transform ? a.heads : 0) + (a.tied ? 1 : 2) * a.kv_heads);
    if (items <= 0) return 0;
    const unsigned blocks = (unsigned)((items + 3) / 4);
    const bool vectors = dtype == KIDI_BF16 && items < (1LL << 30) && (!a.value_dim || a.value_dim == a.head_dim) && !((uintptr_t)a.q_norm & 15) &&
                         !((uintptr_t)a.k_norm & 15) && !(a.head_dim & 7) && !(a.ld & 7) && !((uintptr_t)a.qkv & 15) &&
                         !((uintptr_t)a.k_cache & 15) && !((uintptr_t)a.v_cache & 15) && !((uintptr_t)a.k_normed & 15) &&
                         !(a.ld_k_normed & 7) &&
                         (!a.cos_table || (!(a.rotary_dim & 15) && !((uintptr_t)a.cos_table & 15) &&
                                           !((uintptr_t)a.sin_table & 15)));
    if (vectors) {
        int group_lanes = 1;                    // lanes that cover a head in 16-byte vectors
        while (group_lanes * 8 < a.head_dim) group_lanes <<= 1;
        const long long per_block = 4 * (32 / group_lanes);
        const unsigned vector_blocks = (unsigned)((items + per_block - 1) / per_block);
        if (norm_dtype == KIDI_F32)
            return kidi_launch(rope_store_bf16_kernel<float>, vector_blocks, 128, 0, stream, a, group_lanes);
        if (norm_dtype == KIDI_BF16)
            return kidi_launch(rope_store_bf16_kernel<bf16>, vector_blocks, 128, 0, stream, a, group_lanes);
    }
    if (dtype == KIDI_F32 && norm_dtype == KIDI_F32) return kidi_launch(rope_store_kernel<float, float>, blocks, 128, 0, stream, a);
    if (dtype == KIDI_F32 && norm_dtype == KIDI_BF16) return kidi_launch(rope_store_kernel<float, bf16>, blocks, 128, 0, stream, a);
    if (dtype == KIDI_BF16 && norm_dtype == KIDI_F32) return kidi_launch(rope_store_kernel<bf16, float>, blocks, 128, 0, stream, a);
    if (dtype == KIDI_BF16 && norm_dtype == KIDI_BF16) return kidi_launch(rope_store_kernel<bf16, bf16>, blocks, 128, 0, stream, a);
    return KIDI_REFUSED_DTYPE;
}

// ---------------------------------------------------------------------------
// A norm of a row's whole query (and key) projection, before it is split into heads: all query entries of a row divided by
// their one root mean square and multiplied by a weight of that size, the keys likewise, in place; the keys and the values
// (as they are) also go to the cache where one is given. A block a row; a thread takes V consecutive entries at a time.
struct WideNormArgs {
    void* qkv;                 // [rows, ld]: q heads, k heads, v heads
    long long ld;
    const float* q_norm;       // [heads * head_dim]
    const float* k_norm;       // [kv_heads * head_dim]
    const int* row_seq;        // [rows] (-1: padding row, skipped)
    const int* row_pos;
    const int* seq_slot;
    const int* seq_start;
    const int* seq_len;
    void* k_cache;             // storage of this schedule entry, or null (no write)
    void* v_cache;
    CacheGeometry cache;
    int heads, kv_heads, head_dim, value_dim;
    float eps;
};

constexpr int WIDE_THREADS = 256;

template <typename T, int V> struct Piece;
template <> struct Piece<float, 1> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
    static __device__ __forceinline__ void copy(float* to, const float* from) { *to = *from; }
};
template <> struct Piece<bf16, 1> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[1]) { v[0] = to_float(*p); }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[1]) { *p = from_float<bf16>(v[0]); }
    static __device__ __forceinline__ void copy(bf16* to, const bf16* from) { *to = *from; }
};
template <> struct Piece<bf16, 8> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[8]) { load8(p, v); }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[8]) {
        uint4 packed;
        __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
        for (int i = 0; i < 4; ++i) out[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = packed;
    }
    static __device__ __forceinline__ void copy(bf16* to, const bf16* from) {
        *reinterpret_cast<uint4*>(to) = *reinterpret_cast<const uint4*>(from);
    }
};

template <typename T, int V>
__global__ void __launch_bounds__(WIDE_THREADS) wide_norm_store_kernel(WideNormArgs a) {
    __shared__ float scratch[2][32];
    constexpr int WARPS = WIDE_THREADS / 32;
    constexpr int HELD = V == 8 ? 2 : 1;          // pieces of q that stay in registers between the two passes
    const int row = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    T* q = (T*)a.qkv + row * a.ld;
    const int q_width = a.heads * a.head_dim, k_width = a.kv_heads * a.head_dim, v_width = a.kv_heads * a.value_dim;
    T* k = q + q_width;
    const T* v = k + k_width;
    // (The row's entries are asked for together with its sequence and position; a padding row's are there to be read.)
    const int seq = a.row_seq[row], position = a.row_pos[row];
    float held[HELD][V], held_k[V], piece[V];
    float q_square = 0.f, k_square = 0.f;
    int index = 0;
    for (int c = threadIdx.x * V; c < q_width; c += WIDE_THREADS * V, ++index) {
        Piece<T, V>::load(q + c, piece);
#pragma unroll
        for (int i = 0; i < V; ++i) q_square = fmaf(piece[i], piece[i], q_square);
#pragma unroll
        for (int slot = 0; slot < HELD; ++slot)
            if (slot == index) {
#pragma unroll
                for (int i = 0; i < V; ++i) held[slot][i] = piece[i];
            }
    }
    for (int c = threadIdx.x * V; c < k_width; c += WIDE_THREADS * V) {
        Piece<T, V>::load(k + c, piece);
        if (c < WIDE_THREADS * V) {
#pragma unroll
            for (int i = 0; i < V; ++i) held_k[i] = piece[i];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) k_square = fmaf(piece[i], piece[i], k_square);
    }
    if (seq < 0) return;                              // the same for the whole block
    bool keep = a.k_cache != nullptr;
    if (keep && a.cache.ring_pages)   // a ring keeps the last ring_tokens tokens of the step only
        keep = position >= a.seq_start[seq] + a.seq_len[seq] - (a.cache.ring_pages << a.cache.page_shift);
    const long long offset = keep ? cache_row_offset(a.cache, a.seq_slot[seq], position, 0) : 0;
    const long long key_stride = (long long)a.head_dim << a.cache.page_shift;      // from one head's row to the next head's
    const long long value_stride = (long long)a.value_dim << a.cache.page_shift;
    T* k_cached = (T*)a.k_cache + offset;
    T* v_cached = (T*)a.v_cache + offset / a.head_dim * a.value_dim;
    if (keep)
        for (int c = threadIdx.x * V; c < v_width; c += WIDE_THREADS * V) {
            const int head = c / a.value_dim;
            Piece<T, V>::copy(v_cached + head * value_stride + (c - head * a.value_dim), v + c);
        }
    q_square = warp_sum(q_square);
    k_square = warp_sum(k_square);
    if (lane == 0) { scratch[0][warp] = q_square; scratch[1][warp] = k_square; }
    __syncthreads();
    float q_total = 0.f, k_total = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) { q_total += scratch[0][w]; k_total += scratch[1][w]; }
    const float q_inv = 1.0f / sqrtf(q_total / (float)q_width + a.eps);
    const float k_inv = 1.0f / sqrtf(k_total / (float)k_width + a.eps);
    index = 0;
    for (int c = threadIdx.x * V; c < q_width; c += WIDE_THREADS * V, ++index) {
        if (index >= HELD) Piece<T, V>::load(q + c, piece);
#pragma unroll
        for (int slot = 0; slot < HELD; ++slot)
            if (slot == index) {
#pragma unroll
                for (int i = 0; i < V; ++i) piece[i] = held[slot][i];
            }
#pragma unroll
        for (int i = 0; i < V; ++i) piece[i] = piece[i] * q_inv * a.q_norm[c + i];
        Piece<T, V>::store(q + c, piece);
    }
    for (int c = threadIdx.x * V; c < k_width; c += WIDE_THREADS * V) {
        if (c >= WIDE_THREADS * V) Piece<T, V>::load(k + c, held_k);
#pragma unroll
        for (int i = 0; i < V; ++i) piece[i] = held_k[i] * k_inv * a.k_norm[c + i];
        Piece<T, V>::store(k + c, piece);
        if (keep) {
            const int head = c / a.head_dim;
            Piece<T, V>::store(k_cached + head * key_stride + (c - head * a.head_dim), piece);
        }
    }
}

KIDI_API int kidi_wide_norm_store(const WideNormArgs* args, int rows, int dtype, cudaStream_t stream) {
    const WideNormArgs& a = *args;
    if (rows <= 0) return 0;
    if (a.heads <= 0 || a.kv_heads <= 0 || a.head_dim <= 0 || a.value_dim <= 0 || !a.q_norm || !a.k_norm ||
        (a.k_cache != nullptr) != (a.v_cache != nullptr))
        return KIDI_REFUSED_SIZE;
    const bool vectors = !(a.head_dim & 7) && !(a.value_dim & 7) && !(a.ld & 7) && !((uintptr_t)a.qkv & 15) &&
                         !((uintptr_t)a.k_cache & 15) && !((uintptr_t)a.v_cache & 15);
    if (dtype == KIDI_F32) return kidi_launch(wide_norm_store_kernel<float, 1>, rows, WIDE_THREADS, 0, stream, a);
    if (dtype == KIDI_BF16 && vectors) return kidi_launch(wide_norm_store_kernel<bf16, 8>, rows, WIDE_THREADS, 0, stream, a);
    if (dtype == KIDI_BF16) return kidi_launch(wide_norm_store_kernel<bf16, 1>, rows, WIDE_THREADS, 0, stream, a);
    return KIDI_REFUSED_DTYPE;
}

// ---------------------------------------------------------------------------
struct AttentionArgs {
    const void* q;        // [rows, ldq], head h at h*head_dim
    long long ldq;
    const void* k_step;   // keys of this step's rows [rows, ldkv], kv head g at g*head_dim; null: read the cache only
    const void* v_step;
    long long ldkv;
    const void* k_cache;  // storage of this schedule entry (may be null when every key is in the step)
    const void* v_cache;
    CacheGeometry cache;
    void* out;            // [rows, ldo]
    long long ldo;
    const int* row_seq;   // [rows] (-1: padding row: output zeros)
    const int* row_pos;
    const int* seq_slot;
    const int* seq_start; // tokens in the cache before this step
    const int* seq_row0;  // first packed row of the sequence
    int rows, heads, kv_heads, head_dim, window;  // window 0: every earlier key is visible
    float scale;
    float softcap;        // > 0: a score s becomes softcap * tanh(s / softcap)
    const float* slopes;  // [heads] or null: head h adds slopes[h] * (key position - query position) to a score
    int value_dim;        // width of a value head and of a head of `out` (0: head_dim), at most 256
    const float* sinks;   // [heads] or null: exp(sinks[h]) is added to head h's softmax denominator (a key that
                          // every row sees, with that score as it is, unscaled, and no value)
    const void* gate;     // [rows, ldg] or null: head h of a row is multiplied by sigmoid(gate[row, h])
    long long ldg;
    const float* weight_bias;  // [heads] or null: the weight of a key is sigmoid(score + weight_bias[h]) instead of its
                               // share of a softmax (nothing is normalised over the keys)
    int chunk;                 // > 0: only keys of the query's own run of `chunk` positions are seen
    float out_scale;           // the result is multiplied by it
    int tied;                  // k_step / k_cache hold keys before their norm, which are the values too (v_step, v_cache name
                               // the same rows); a score takes the factor 1 / sqrt(mean square of the key + key_eps)
    float key_eps;
    const float* distance_bias;   // [heads, bias_stride] or null: entry min(p - u, bias_last) of head h's row is added to a score
    int bias_stride, bias_last;
    const void* element_gate;     // [rows, ld_element_gate] or null: the result is multiplied by sigmoid of it, element by element
    long long ld_element_gate;
};

// One block of 4 warps per (row, head). Warp w takes keys lo+w, lo+w+4, ... in
// ascending order with an online softmax; the four partial results are merged in
// warp order. The order depends on the row's position and window only, so a row's
// result is the same in every batch and under every cut of the work.
template <typename T>
__global__ void __launch_bounds__(128) attention_generic_kernel(AttentionArgs a) {
    __shared__ float query[256];
    __shared__ float part_acc[4][256];
    __shared__ float part_max[4], part_sum[4];
    const int row = blockIdx.x, head = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int d = a.head_dim;
    const int vd = a.value_dim ? a.value_dim : d;
    T* out = (T*)a.out + row * a.ldo + (long long)head * vd;
    const int seq = a.row_seq[row];
    if (seq < 0) {
        for (int c = threadIdx.x; c < vd; c += 128) out[c] = from_float<T>(0.f);
        return;
    }
    const int position = a.row_pos[row];
    const int first = first_visible(position, a.window, a.chunk);
    const int kv_head = head / (a.heads / a.kv_heads);
    const int slot = a.seq_slot[seq];
    const int start = a.k_step ? a.seq_start[seq] : 0x7fffffff;  // keys >= start come from the step
    const int row0 = a.seq_row0[seq];
    const T* q = (const T*)a.q + row * a.ldq + (long long)head * d;
    for (int c = threadIdx.x; c < d; c += 128) query[c] = to_float(q[c]);
    __syncthreads();

    float best = -INFINITY, denom = 0.f;
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = 0.f;
    for (int u = first + warp; u <= position; u += 4) {
        const T *key, *value;
        if (u >= start) {
            const long long offset = (long long)(row0 + u - start) * a.ldkv;
            key = (const T*)a.k_step + offset + (long long)kv_head * d;
            value = (const T*)a.v_step + offset + (long long)kv_head * vd;
        } else {
            const long long offset = cache_row_offset(a.cache, slot, u, kv_head);
            key = (const T*)a.k_cache + offset;
            value = (const T*)a.v_cache + offset / d * vd;
        }
        float dot = 0.f, square = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            if (c < d) {
                const float entry = to_float(key[c]);
                dot = fmaf(query[c], entry, dot);
                square = fmaf(entry, entry, square);
            }
        }
        float score = warp_sum(dot) * a.scale;
        if (a.tied) score *= 1.0f / sqrtf(warp_sum(square) / (float)d + a.key_eps);
        if (a.softcap > 0.f) score = a.softcap * tanhf(score / a.softcap);
        if (a.slopes) score += a.slopes[head] * (float)(u - position);
        if (a.distance_bias) score += a.distance_bias[(long long)head * a.bias_stride + min(position - u, a.bias_last)];
        if (a.weight_bias) {             // a weight of its own for every key: nothing to rescale
            const float weight = 1.0f / (1.0f + expf(-(score + a.weight_bias[head])));
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int c = lane + 32 * i;
                if (c < vd) acc[i] = fmaf(weight, to_float(value[c]), acc[i]);
            }
            continue;
        }
        const float next = fmaxf(best, score);
        const float keep = expf(best - next);  // 0 on the first key (best = -inf)
        const float weight = expf(score - next);
        denom = denom * keep + weight;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = lane + 32 * i;
            if (c < vd) acc[i] = acc[i] * keep + weight * to_float(value[c]);
        }
        best = next;
    }
    if (lane == 0) { part_max[warp] = best; part_sum[warp] = denom; }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < vd) part_acc[warp][c] = acc[i];
    }
    __syncthreads();
    float top = part_max[0];
#pragma unroll
    for (int w = 1; w < 4; ++w) top = fmaxf(top, part_max[w]);
    const float sink = a.sinks ? a.sinks[head] : -INFINITY;
    top = fmaxf(top, sink);
    float total = a.sinks ? expf(sink - top) : 0.f, factor[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) {
        factor[w] = part_max[w] == -INFINITY ? 0.f : expf(part_max[w] - top);
        total += part_sum[w] * factor[w];
    }
    if (a.weight_bias) {
        total = 1.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) factor[w] = 1.f;
    }
    float gate = 1.f;
    if (a.gate) gate = 1.0f / (1.0f + expf(-to_float(((const T*)a.gate)[row * a.ldg + head])));
    for (int c = threadIdx.x; c < vd; c += 128) {
        float value = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) value += part_acc[w][c] * factor[w];
        value /= total;
        if (a.gate) value *= gate;
        if (a.element_gate)
            value *= 1.0f / (1.0f + expf(-to_float(((const T*)a.element_gate)[row * a.ld_element_gate + (long long)head * vd + c])));
        out[c] = from_float<T>(value * a.out_scale);
    }
}

KIDI_API int kidi_attention_generic(const AttentionArgs* args, int dtype, cudaStream_t stream) {
    const AttentionArgs& a = *args;
    if (a.rows <= 0) return 0;
    if (a.head_dim > 256 || a.head_dim <= 0 || a.heads % a.kv_heads || a.heads > 65535 || a.value_dim < 0 ||
        a.value_dim > 256 || a.chunk < 0 || (a.weight_bias && a.sinks) || (a.tied && a.value_dim && a.value_dim != a.head_dim) ||
        (a.distance_bias && (a.bias_last < 0 || a.bias_stride <= a.bias_last)))
        return KIDI_REFUSED_SIZE;
    dim3 grid(a.rows, a.heads);
    if (dtype == KIDI_F32) return kidi_launch(attention_generic_kernel<float>, grid, 128, 0, stream, a);
    if (dtype == KIDI_BF16) return kidi_launch(attention_generic_kernel<bf16>, grid, 128, 0, stream, a);
    return KIDI_REFUSED_DTYPE;
}
