// Linear attention with one fixed decay per head ("lightning attention") around a 32-bit state:
//
//     S_t = decay_h S_(t-1) + k_t v_t^T            S: [dim, vdim] per head
//     o_t = S_t^T q_t
//
// with q, k and v as their projections' activations left them. What is here beside the scan that other recurrences
// with one decay per head share (scalar_recurrence.cu):
//
//  * one token a sequence (decoding): a block takes 32 columns of a (sequence, head), reads its part of the state
//    once with every load in flight, writes it back and adds up the read-out;
//  * the finish: a row's concatenated heads divided by their one root mean square, times a weight, times
//    sigmoid(gate), times a number;
//  * SiLU on a range of a projection's columns, in place.
//
// State, decay, read-out and norm are 32-bit.
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

// V columns a thread (4 where the widths allow 16-byte accesses), 32 / V threads beside one another, the others on
// further state rows; DEPTH rows a thread are in flight together.
template <typename T, int V>
__global__ void __launch_bounds__(THREADS) linear_step_kernel(LinearStepArgs a) {
    typedef typename Columns<V>::type Vec;
    constexpr int LANES = COLUMNS / V, ROWS = THREADS / LANES, DEPTH = 4;
    extern __shared__ __align__(16) float shared[];        // keys [dim], queries [dim], then partial sums [ROWS][COLUMNS]
    float* keys = shared;
    float* queries = shared + a.dim;
    float* partial = shared + ((2 * a.dim + 3) & ~3);
    const int head = blockIdx.y, seq = blockIdx.x;
    const int row = a.seq_row0[seq];
    if (a.row_seq[row] < 0) return;                        // a padding sequence touches no state
    const int dim = a.dim, vdim = a.vdim;
    const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES;
    const int column = blockIdx.z * COLUMNS + lane * V;
    const bool live = column < vdim;                       // (vdim is a multiple of V)
    float* state = a.state + ((long long)a.seq_slot[seq] * a.heads + head) * dim * vdim + column;
    Vec s[DEPTH];
#pragma unroll
    for (int j = 0; j < DEPTH; ++j) {
        const int d = group + j * ROWS;
        if (live && d < dim) s[j] = *reinterpret_cast<const Vec*>(state + (long long)d * vdim);
    }
    for (int d = threadIdx.x; d < dim; d += THREADS) {
        keys[d] = to_float(((const T*)a.k)[row * a.ldk + (long long)head * dim + d]);
        queries[d] = to_float(((const T*)a.q)[row * a.ldq + (long long)head * dim + d]);
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
    if (threadIdx.x < COLUMNS && blockIdx.z * COLUMNS + threadIdx.x < vdim) {
        float read = 0.f;
#pragma unroll
        for (int g = 0; g < ROWS; ++g) read += partial[g * COLUMNS + threadIdx.x];
        a.out[((long long)row * a.heads + head) * vdim + blockIdx.z * COLUMNS + threadIdx.x] = read;
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
    if (a.heads <= 0 || a.heads > 65535 || a.dim <= 0 || a.vdim <= 0 || spans > 65535 || shared > 48 * 1024)
        return KIDI_REFUSED_SIZE;
    const dim3 grid(a.seqs, a.heads, spans);
    const bool vectors = !(a.vdim & 3) && !((uintptr_t)a.state & 15);
    if (dtype == KIDI_F32)
        return vectors ? kidi_launch(linear_step_kernel<float, 4>, grid, THREADS, shared, stream, a)
                       : kidi_launch(linear_step_kernel<float, 1>, grid, THREADS, shared, stream, a);
    if (dtype == KIDI_BF16)
        return vectors ? kidi_launch(linear_step_kernel<bf16, 4>, grid, THREADS, shared, stream, a)
                       : kidi_launch(linear_step_kernel<bf16, 1>, grid, THREADS, shared, stream, a);
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
