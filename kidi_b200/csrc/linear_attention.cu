// Linear attention with one fixed decay per head ("lightning attention") around a 32-bit state:
//
//     S_t = decay_h S_(t-1) + k_t v_t^T            S: [dim, vdim] per head
//     o_t = S_t^T q_t
//
// with q, k and v as their projections' activations left them, or with q and k rotated by position and k times a number
// ("retention"; both in 32-bit, on the way into the recurrence). What is here beside the scan that other recurrences
// with one decay per head share (scalar_recurrence.cu):
//
//  * one token a sequence (decoding): a block takes 32 columns of a (sequence, head), reads its part of the state
//    once with every load in flight, writes it back and adds up the read-out. The blocks of a head can form a cluster
//    that also finishes the head: divided by its root mean square (the blocks exchange their sums of squares through
//    distributed shared memory), times the SiLU or sigmoid of a gate, rounded;
//  * rotated and scaled queries and keys as 32-bit numbers (for the scan);
//  * the finish head by head as a kernel of its own;
//  * the finish: a row's concatenated heads divided by their one root mean square, times a weight, times
//    sigmoid(gate), times a number;
//  * SiLU on a range of a projection's columns, in place.
//
// State, decay, read-out and norm are 32-bit.
#include <cooperative_groups.h>

#include "common.cuh"

struct LinearStepArgs {
    const void* q;         // [rows, ldq]: head h at h * dim
    long long ldq;
    const void* k;
    long long ldk;
    const void* v;         // [rows, ldv]: head h at h * vdim
    long long ldv;
    const float* decay;    // [heads]
    float* state;          // [slots + 1, heads, dim, vdim]
    float* out;            // [rows, heads * vdim]
    const int* row_seq;    // [rows] (-1: padding)
    const int* seq_slot;   // [seqs]
    const int* seq_row0;   // [seqs]
    int seqs, heads, dim, vdim;
    // Optional: entries i and i + rotary_dim / 2 of a head's q and k (i < rotary_dim / 2) are turned by position, and k is
    // multiplied by key_scale.
    const float* cos_table;   // [positions, rotary_dim / 2] or null
    const float* sin_table;
    const int* row_pos;       // [rows]
    int rotary_dim;
    float key_scale;
    // Optional: the head is finished here. `finished` (of the step's element type) takes read / rms(read) * act(gate).
    const void* gate;         // [rows, ldg] or null: head h at h * vdim
    long long ldg;
    void* finished;           // [rows, ldf]
    long long ldf;
    float eps;
    int gate_silu;            // act: 1 SiLU, 0 sigmoid
};

namespace {

constexpr int THREADS = 256;
constexpr int COLUMNS = 32;                        // state columns of a block of the one-token kernel

template <int V> struct Columns;
template <> struct Columns<4> { typedef float4 type; };
template <> struct Columns<1> { typedef float type; };

__device__ __forceinline__ void dot_add(float4& s, float keep, float key, const float4& v, float query, float4& sum) {
    s.x = fmaf(keep, s.x, key * v.x); s.y = fmaf(keep, s.y, key * v.y);
    s.z = fmaf(keep, s.z, key * v.z); s.w = fmaf(keep, s.w, key * v.w);
    sum.x = fmaf(s.x, query, sum.x); sum.y = fmaf(s.y, query, sum.y);
    sum.z = fmaf(s.z, query, sum.z); sum.w = fmaf(s.w, query, sum.w);
}
__device__ __forceinline__ void dot_add(float& s, float keep, float key, const float& v, float query, float& sum) {
    s = fmaf(keep, s, key * v);
    sum = fmaf(s, query, sum);
}

// Entry d of a head's row x, rotated.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int d, const float* cos_table, const float* sin_table, int rotary_dim,
                                         int position) {
    const float own = to_float(x[d]);
    if (d >= rotary_dim) return own;
    const int half = rotary_dim / 2, j = d < half ? d : d - half;
    const float other = to_float(x[d < half ? d + half : d - half]);
    const float cosine = cos_table[(long long)position * half + j], sine = sin_table[(long long)position * half + j];
    return own * cosine + (d < half ? -other : other) * sine;
}

__device__ __forceinline__ float gate_activation(float z, int silu) {
    const float s = 1.0f / (1.0f + expf(-z));
    return silu ? z * s : s;
}

// V columns a thread (4 where the widths allow 16-byte accesses), 32 / V threads beside one another, the others on
// further state rows; DEPTH rows a thread are in flight together.
// FINISH: the grid's blocks along x (a head's columns) form a cluster and finish the head.
template <typename T, int V, bool FINISH>
__global__ void __launch_bounds__(THREADS) linear_step_kernel(LinearStepArgs a) {
    typedef typename Columns<V>::type Vec;
    constexpr int LANES = COLUMNS / V, ROWS = THREADS / LANES, DEPTH = 4;
    extern __shared__ __align__(16) float shared[];        // keys [dim], queries [dim], then partial sums [ROWS][COLUMNS]
    float* keys = shared;
    float* queries = shared + a.dim;
    float* partial = shared + ((2 * a.dim + 3) & ~3);
    __shared__ float squares[8];                           // of the head's columns, by block of the cluster
    const int head = blockIdx.y, seq = blockIdx.z;
    const int row = a.seq_row0[seq];
    if (a.row_seq[row] < 0) return;                        // a padding sequence touches no state (nor does its whole cluster)
    const int dim = a.dim, vdim = a.vdim;
    const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES;
    // (Every block of a cluster has begun before another one writes to its shared memory.)
    if constexpr (FINISH) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    const int column = blockIdx.x * COLUMNS + lane * V;
    const bool live = column < vdim;                       // (vdim is a multiple of V)
    float* state = a.state + ((long long)a.seq_slot[seq] * a.heads + head) * dim * vdim + column;
    Vec s[DEPTH];
#pragma unroll
    for (int j = 0; j < DEPTH; ++j) {
        const int d = group + j * ROWS;
        if (live && d < dim) s[j] = *reinterpret_cast<const Vec*>(state + (long long)d * vdim);
    }
    const int rotary_dim = a.cos_table ? a.rotary_dim : 0, position = a.cos_table ? a.row_pos[row] : 0;
    for (int d = threadIdx.x; d < dim; d += THREADS) {
        keys[d] = a.key_scale * rotated((const T*)a.k + row * a.ldk + (long long)head * dim, d, a.cos_table, a.sin_table, rotary_dim, position);
        queries[d] = rotated((const T*)a.q + row * a.ldq + (long long)head * dim, d, a.cos_table, a.sin_table, rotary_dim, position);
    }
    float value[V], total[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
        value[e] = live ? to_float(((const T*)a.v)[row * a.ldv + (long long)head * vdim + column + e]) : 0.f;
        total[e] = 0.f;
    }
    const Vec v = *reinterpret_cast<const Vec*>(value);
    Vec sum = *reinterpret_cast<const Vec*>(total);
    const float keep = a.decay[head];
    __syncthreads();
    for (int base = 0; base < dim; base += DEPTH * ROWS) {
        if (base > 0) {
#pragma unroll
            for (int j = 0; j < DEPTH; ++j) {
                const int d = base + group + j * ROWS;
                if (live && d < dim) s[j] = *reinterpret_cast<const Vec*>(state + (long long)d * vdim);
            }
        }
#pragma unroll
        for (int j = 0; j < DEPTH; ++j) {
            const int d = base + group + j * ROWS;
            if (live && d < dim) {
                dot_add(s[j], keep, keys[d], v, queries[d], sum);
                *reinterpret_cast<Vec*>(state + (long long)d * vdim) = s[j];
            }
        }
    }
    *reinterpret_cast<Vec*>(partial + group * COLUMNS + lane * V) = sum;
    __syncthreads();
    float read = 0.f;
    const int mine = blockIdx.x * COLUMNS + threadIdx.x;     // the column that a thread of the first warp finishes
    const bool reads = threadIdx.x < COLUMNS && mine < vdim;
    if (reads) {
#pragma unroll
        for (int g = 0; g < ROWS; ++g) read += partial[g * COLUMNS + threadIdx.x];
        if (!FINISH) a.out[((long long)row * a.heads + head) * vdim + mine] = read;
    }
    if constexpr (FINISH) {
        cooperative_groups::cluster_group cluster = cooperative_groups::this_cluster();
        const int blocks = gridDim.x;                        // == the cluster's size, <= 8
        float z = 0.f;
        asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
        if (reads) z = to_float(((const T*)a.gate)[row * a.ldg + (long long)head * vdim + mine]);
        if (threadIdx.x < 32) {
            const float square = warp_sum(read * read);      // (threads without a column hold zero)
            if (threadIdx.x < blocks) *cluster.map_shared_rank(&squares[blockIdx.x], threadIdx.x) = square;
        }
        cluster.sync();                                      // nothing is read from another block after it
        if (reads) {
            float total = 0.f;
            for (int b = 0; b < blocks; ++b) total += squares[b];
            ((T*)a.finished)[row * a.ldf + (long long)head * vdim + mine] =
                from_float<T>(read / sqrtf(total / (float)vdim + a.eps) * gate_activation(z, a.gate_silu));
        }
    }
}

// Rotated queries and keys (keys times key_scale) and values, all as 32-bit numbers: out[r] = [q | k | v]. A block a row.
template <typename T>
__global__ void __launch_bounds__(THREADS)
rotate_heads_kernel(const T* __restrict__ q, long long ldq, const T* __restrict__ k, long long ldk, const T* __restrict__ v,
                    long long ldv, float* __restrict__ out, const float* __restrict__ cos_table,
                    const float* __restrict__ sin_table, const int* __restrict__ row_pos, int rotary_dim, float key_scale,
                    int heads, int dim, int vdim) {
    const long long row = blockIdx.x;
    const int qk = heads * dim, values = heads * vdim, position = row_pos[row];
    float* to = out + row * (2 * qk + values);
    for (int c = threadIdx.x; c < qk; c += THREADS) {
        const int head = c / dim, d = c - head * dim;
        to[c] = rotated(q + row * ldq + head * dim, d, cos_table, sin_table, rotary_dim, position);
        to[qk + c] = key_scale * rotated(k + row * ldk + head * dim, d, cos_table, sin_table, rotary_dim, position);
    }
    for (int c = threadIdx.x; c < values; c += THREADS) to[2 * qk + c] = to_float(v[row * ldv + c]);
}

// y = read / sqrt(mean(read^2) + eps) * weight * act(gate) * factor head by head (weight: [heads * vdim] or null). A warp a
// (row, head).
template <typename T>
__global__ void __launch_bounds__(THREADS)
head_gate_kernel(const float* __restrict__ read, const float* __restrict__ weight, const T* __restrict__ gate, long long ldg,
                 T* __restrict__ out, long long ldo, long long items, int heads, int vdim, float eps, float factor, int silu) {
    const long long item = (long long)blockIdx.x * (THREADS / 32) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= items) return;
    const long long row = item / heads;
    const int head = (int)(item - row * heads);
    const float* source = read + item * vdim;
    float square = 0.f;
    for (int c = lane; c < vdim; c += 32) square = fmaf(source[c], source[c], square);
    const float inv = factor / sqrtf(warp_sum(square) / (float)vdim + eps);
    for (int c = lane; c < vdim; c += 32) {
        const int at = head * vdim + c;
        const float y = source[c] * inv * gate_activation(to_float(gate[row * ldg + at]), silu);
        out[row * ldo + at] = from_float<T>(weight ? y * weight[at] : y);
    }
}

// A block a row: y = read / sqrt(mean(read^2) + eps) * weight * sigmoid(gate) * factor over all of the row's heads.
template <typename T>
__global__ void __launch_bounds__(THREADS)
normed_gate_kernel(const float* __restrict__ read, const float* __restrict__ weight, const T* __restrict__ gate, long long ldg,
                   T* __restrict__ out, long long ldo, int width, float eps, float factor) {
    __shared__ float scratch[32];
    const long long row = blockIdx.x;
    const float* source = read + row * width;
    float square = 0.f;
    for (int c = threadIdx.x; c < width; c += THREADS) square = fmaf(source[c], source[c], square);
    const float inv = factor / sqrtf(block_sum<THREADS>(square, scratch) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += THREADS)
        out[row * ldo + c] = from_float<T>(source[c] * inv * weight[c] / (1.0f + expf(-to_float(gate[row * ldg + c]))));
}

// y sigmoid(z) with the fast exponential and division (a few units in the last place; for results that are rounded to
// bfloat16; far below zero the exponential is held at 2^115, so that the quotient stays a number).
__device__ __forceinline__ float sigmoid_times(float y, float z) {
    return __fdividef(y, 1.0f + __expf(fminf(-z, 80.f)));
}

// The same for bfloat16 results of widths that are multiples of 4, from 16-byte pieces of the read-out; up to HELD
// pieces a thread stay in registers between the two passes.
__global__ void __launch_bounds__(THREADS)
normed_gate_bf16x4_kernel(const float* __restrict__ read, const float* __restrict__ weight, const bf16* __restrict__ gate,
                          long long ldg, bf16* __restrict__ out, long long ldo, int width, float eps, float factor) {
    __shared__ float scratch[32];
    constexpr int HELD = 4;
    const long long row = blockIdx.x;
    const float4* source = reinterpret_cast<const float4*>(read + row * width);
    const int pieces = width >> 2;
    float4 held[HELD];
    float square = 0.f;
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
        const int c = threadIdx.x + i * THREADS;
        held[i] = c < pieces ? source[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
        square = fmaf(held[i].x, held[i].x, square);
        square = fmaf(held[i].y, held[i].y, square);
        square = fmaf(held[i].z, held[i].z, square);
        square = fmaf(held[i].w, held[i].w, square);
    }
    for (int c = threadIdx.x + HELD * THREADS; c < pieces; c += THREADS) {
        const float4 x = source[c];
        square = fmaf(x.x, x.x, square);
        square = fmaf(x.y, x.y, square);
        square = fmaf(x.z, x.z, square);
        square = fmaf(x.w, x.w, square);
    }
    const float inv = factor / sqrtf(block_sum<THREADS>(square, scratch) / (float)width + eps);
    auto write = [&](int c, const float4& x) {
        const float4 w = reinterpret_cast<const float4*>(weight)[c];
        const uint2 raw = *reinterpret_cast<const uint2*>(gate + row * ldg + 4 * c);
        const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        uint2 packed;
        *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(sigmoid_times(x.x * inv * w.x, g0.x),
                                                                             sigmoid_times(x.y * inv * w.y, g0.y));
        *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(sigmoid_times(x.z * inv * w.z, g1.x),
                                                                             sigmoid_times(x.w * inv * w.w, g1.y));
        *reinterpret_cast<uint2*>(out + row * ldo + 4 * c) = packed;
    };
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c < pieces) write(c, held[i]);
    }
    for (int c = threadIdx.x + HELD * THREADS; c < pieces; c += THREADS) write(c, source[c]);
}

// x[r, begin : begin + width] <- silu of itself.
template <typename T>
__global__ void silu_columns_kernel(T* __restrict__ x, long long ld, long long total, int begin, int width) {
    const long long index = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (index >= total) return;
    const long long row = index / width;
    T* at = x + row * ld + begin + (index - row * width);
    const float z = to_float(*at);
    *at = from_float<T>(z / (1.0f + expf(-z)));
}
__global__ void silu_columns_bf16x8_kernel(bf16* __restrict__ x, long long ld, long long groups, int begin, int width) {
    const long long index = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (index >= groups) return;
    const int per_row = width >> 3;
    const long long row = index / per_row;
    bf16* at = x + row * ld + begin + (index - row * per_row) * 8;
    uint4 raw = *reinterpret_cast<const uint4*>(at);
    __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 z = __bfloat1622float2(pairs[i]);
        pairs[i] = __floats2bfloat162_rn(sigmoid_times(z.x, z.x), sigmoid_times(z.y, z.y));
    }
    *reinterpret_cast<uint4*>(at) = raw;
}

}  // namespace

KIDI_API int kidi_linear_step(const LinearStepArgs* args, int dtype, cudaStream_t stream) {
    const LinearStepArgs& a = *args;
    if (a.seqs <= 0) return 0;
    const int spans = (a.vdim + COLUMNS - 1) / COLUMNS;
    const size_t shared = (size_t)(((2 * a.dim + 3) & ~3) + THREADS * 4) * sizeof(float);    // ROWS * COLUMNS = THREADS * V
    if (a.heads <= 0 || a.heads > 65535 || a.seqs > 65535 || a.dim <= 0 || a.vdim <= 0 || shared > 48 * 1024 ||
        (a.cos_table && (!a.sin_table || !a.row_pos || (a.rotary_dim & 1) || a.rotary_dim < 0 || a.rotary_dim > a.dim)) ||
        (a.gate && (spans > 8 || !a.finished)) || (!a.gate && !a.out))
        return KIDI_REFUSED_SIZE;
    const dim3 grid(spans, a.heads, a.seqs);
    const bool vectors = !(a.vdim & 3) && !((uintptr_t)a.state & 15);
#define KIDI_CASE(D, T)                                                                                                     \
    if (dtype == D) {                                                                                                       \
        if (a.gate)                                                                                                         \
            return vectors ? kidi_launch_clusters(linear_step_kernel<T, 4, true>, grid, THREADS, shared, stream, spans, a)  \
                           : kidi_launch_clusters(linear_step_kernel<T, 1, true>, grid, THREADS, shared, stream, spans, a); \
        return vectors ? kidi_launch(linear_step_kernel<T, 4, false>, grid, THREADS, shared, stream, a)                     \
                       : kidi_launch(linear_step_kernel<T, 1, false>, grid, THREADS, shared, stream, a);                    \
    }
    KIDI_CASE(KIDI_F32, float)
    KIDI_CASE(KIDI_BF16, bf16)
#undef KIDI_CASE
    return KIDI_REFUSED_DTYPE;
}

KIDI_API int kidi_rotate_heads(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, int dtype,
                               float* out, const float* cos_table, const float* sin_table, const int* row_pos, int rotary_dim,
                               float key_scale, int rows, int heads, int dim, int vdim, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || dim <= 0 || vdim <= 0 || rotary_dim < 0 || (rotary_dim & 1) || rotary_dim > dim || !row_pos ||
        (rotary_dim > 0 && (!cos_table || !sin_table)))
        return KIDI_REFUSED_SIZE;
    if (dtype == KIDI_F32)
        return kidi_launch(rotate_heads_kernel<float>, rows, THREADS, 0, stream, (const float*)q, ldq, (const float*)k, ldk,
                           (const float*)v, ldv, out, cos_table, sin_table, row_pos, rotary_dim, key_scale, heads, dim, vdim);
    if (dtype == KIDI_BF16)
        return kidi_launch(rotate_heads_kernel<bf16>, rows, THREADS, 0, stream, (const bf16*)q, ldq, (const bf16*)k, ldk,
                           (const bf16*)v, ldv, out, cos_table, sin_table, row_pos, rotary_dim, key_scale, heads, dim, vdim);
    return KIDI_REFUSED_DTYPE;
}

KIDI_API int kidi_head_norm_gate(const float* read, const float* weight, const void* gate, long long ldg, int dtype, void* out,
                                 long long ldo, int rows, int heads, int vdim, float eps, float factor, int silu,
                                 cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || vdim <= 0) return KIDI_REFUSED_SIZE;
    const long long items = (long long)rows * heads;
    const unsigned blocks = (unsigned)((items + THREADS / 32 - 1) / (THREADS / 32));
    if (dtype == KIDI_F32)
        return kidi_launch(head_gate_kernel<float>, blocks, THREADS, 0, stream, read, weight, (const float*)gate, ldg, (float*)out,
                           ldo, items, heads, vdim, eps, factor, silu);
    if (dtype == KIDI_BF16)
        return kidi_launch(head_gate_kernel<bf16>, blocks, THREADS, 0, stream, read, weight, (const bf16*)gate, ldg, (bf16*)out, ldo,
                           items, heads, vdim, eps, factor, silu);
    return KIDI_REFUSED_DTYPE;
}

KIDI_API int kidi_normed_gate(const float* read, const float* weight, const void* gate, long long ldg, int dtype, void* out,
                              long long ldo, int rows, int width, float eps, float factor, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (width <= 0) return KIDI_REFUSED_SIZE;
    if (dtype == KIDI_F32)
        return kidi_launch(normed_gate_kernel<float>, rows, THREADS, 0, stream, read, weight, (const float*)gate, ldg,
                           (float*)out, ldo, width, eps, factor);
    if (dtype != KIDI_BF16) return KIDI_REFUSED_DTYPE;
    if (!(width & 3) && !(ldg & 3) && !(ldo & 3) && !((uintptr_t)read & 15) && !((uintptr_t)weight & 15) &&
        !((uintptr_t)gate & 7) && !((uintptr_t)out & 7))
        return kidi_launch(normed_gate_bf16x4_kernel, rows, THREADS, 0, stream, read, weight, (const bf16*)gate, ldg,
                           (bf16*)out, ldo, width, eps, factor);
    return kidi_launch(normed_gate_kernel<bf16>, rows, THREADS, 0, stream, read, weight, (const bf16*)gate, ldg, (bf16*)out,
                       ldo, width, eps, factor);
}

KIDI_API int kidi_silu_columns(void* x, long long ld, int dtype, int rows, int begin, int width, cudaStream_t stream) {
    const long long total = (long long)rows * width;
    if (total <= 0) return 0;
    if (begin < 0) return KIDI_REFUSED_SIZE;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == KIDI_F32) return kidi_launch(silu_columns_kernel<float>, blocks, 256, 0, stream, (float*)x, ld, total, begin, width);
    if (dtype != KIDI_BF16) return KIDI_REFUSED_DTYPE;
    if (!(width & 7) && !(begin & 7) && !(ld & 7) && !((uintptr_t)x & 15))
        return kidi_launch(silu_columns_bf16x8_kernel, (unsigned)(((total >> 3) + 255) / 256), 256, 0, stream, (bf16*)x, ld,
                           total >> 3, begin, width);
    return kidi_launch(silu_columns_kernel<bf16>, blocks, 256, 0, stream, (bf16*)x, ld, total, begin, width);
}
