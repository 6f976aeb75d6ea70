// Linear attention with one fixed decay per head over many tokens (prompts), in chunks of 64 tokens on the tensor cores,
// compiled for one pair of head widths (-DKIDI_LINEAR_DIM=..., -DKIDI_LINEAR_VDIM=..., multiples of 16 up to 256).
//
// With a the head's decay, tokens 0 .. n-1 of a chunk and S the state before it,
//
//     o_i = a^(i+1) S^T q_i + sum over j <= i of a^(i-j) (q_i . k_j) v_j
//     S'  = a^n S + sum over j of a^(n-1-j) k_j v_j^T
//
// in three kernels: the sum of the second line for every chunk of every head at once; the states before the chunks, an
// element-wise walk over a head's chunks; and the first line for every chunk at once.
//
// The recurrence is 32-bit although its products run on bfloat16 tensor cores: q, k and v come as bfloat16 numbers, and
// every 32-bit factor (decayed keys, decayed scores, the state) enters as three bfloat16 numbers whose sum is the 32-bit
// number to the last bit or nearly (8 + 8 + 8 significant bits), each multiplied into the same 32-bit accumulators. States
// and their walk are 32-bit throughout.
//
// mma.sync serves these products, not tcgen05: they are 64 x 64 x dim and dim x vdim x 64 with factors that are made in
// registers (decays, splits), which an mma.sync operand is and a tcgen05 operand is not (it would have to go through
// shared memory three times over).
#include "common.cuh"

#ifndef KIDI_LINEAR_DIM
#error "compile with -DKIDI_LINEAR_DIM=<query/key head width> -DKIDI_LINEAR_VDIM=<value head width>"
#endif

struct LinearChunksArgs {
    const bf16* q;          // [rows, ldq]: head h at h * dim
    long long ldq;
    const bf16* k;
    long long ldk;
    const bf16* v;          // [rows, ldv]: head h at h * vdim
    long long ldv;
    const float* decay;     // [heads]
    float* state;           // [slots + 1, heads, dim, vdim]
    float* out;             // [rows, heads * vdim]
    float* sums;            // [chunks, group, dim, vdim]: a chunk's own sum
    bf16* before;           // [chunks, group, 3, dim, vdim]: the state before a chunk, in three parts
    const int* row_seq;     // [rows] (-1: padding)
    const int* seq_slot;    // [seqs]
    const int* seq_row0;    // [seqs]
    const int* seq_len;     // [seqs]
    int seqs, heads;
    int head0, group;       // the heads of this launch: head0 .. head0 + group - 1
    int max_chunks;         // chunks of the longest sequence
};

namespace {

constexpr int D = KIDI_LINEAR_DIM, E = KIDI_LINEAR_VDIM;
static_assert(D % 16 == 0 && E % 16 == 0 && D >= 16 && E >= 16 && D <= 256 && E <= 256, "head widths: multiples of 16 up to 256");
constexpr int CHUNK = 64;
constexpr int THREADS = 256;
constexpr int DP = D + 8, EP = E + 8;               // row pitches: ldmatrix without bank conflicts
constexpr int SLICE = D % 32 == 0 ? 32 : 16;        // rows of the state that are in shared memory at a time
constexpr int SLICES = D / SLICE;

// A sequence's chunks follow one another; the first one's index (no two sequences overlap: a chunk index grows by at
// least the sequence's chunks between neighbours).
__device__ __forceinline__ int first_chunk(int row0, int seq) { return row0 / CHUNK + seq; }

__device__ __forceinline__ unsigned smem_address(const void* pointer) { return (unsigned)__cvta_generic_to_shared(pointer); }
__device__ __forceinline__ void copy_async_16(void* shared, const void* global, bool valid) {
    const int bytes = valid ? 16 : 0;               // 0: zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_address(shared)), "l"(global), "r"(bytes));
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;"); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* shared) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_address(shared)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* shared) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_address(shared)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Two 32-bit numbers as three pairs of bfloat16 numbers that add up to them.
__device__ __forceinline__ void split_pair(float x, float y, unsigned& first, unsigned& second, unsigned& third) {
    __nv_bfloat162 pair = __floats2bfloat162_rn(x, y);
    first = *reinterpret_cast<unsigned*>(&pair);
    float2 back = __bfloat1622float2(pair);
    x -= back.x; y -= back.y;
    pair = __floats2bfloat162_rn(x, y);
    second = *reinterpret_cast<unsigned*>(&pair);
    back = __bfloat1622float2(pair);
    pair = __floats2bfloat162_rn(x - back.x, y - back.y);
    third = *reinterpret_cast<unsigned*>(&pair);
}

__device__ __forceinline__ float2 unpack(unsigned pair) { return __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&pair)); }

// The chunk's rows of q, k or v (WIDTH columns from `source`, row stride ld) into shared memory; rows past the end: zeros.
template <int WIDTH>
__device__ __forceinline__ void load_rows(bf16* tile, const bf16* source, long long ld, int tokens) {
    constexpr int PIECES = WIDTH / 8, PITCH = WIDTH + 8;
    for (int i = threadIdx.x; i < CHUNK * PIECES; i += THREADS) {
        const int r = i / PIECES, c = i - r * PIECES;
        const bool valid = r < tokens;
        copy_async_16(tile + r * PITCH + c * 8, source + (long long)(valid ? r : 0) * ld + c * 8, valid);
    }
}

struct Chunk {
    int tokens, row, index;          // of the chunk: its tokens, its first row, its place in the scratch memory
    bool live;
    __device__ __forceinline__ Chunk(const LinearChunksArgs& a, int seq, int number) {
        const int row0 = a.seq_row0[seq], count = a.seq_len[seq];
        live = number * CHUNK < count && a.row_seq[row0] >= 0;
        tokens = min(CHUNK, count - number * CHUNK);
        row = row0 + number * CHUNK;
        index = first_chunk(row0, seq) + number;
    }
};

// ---------------------------------------------------------------- a chunk's own sum
// [dim, vdim] = sum over j of a^(n-1-j) k_j v_j^T. A warp takes 16 rows (of dim) by up to 64 columns (of vdim) at a time;
// the keys come transposed out of shared memory, are decayed and split in registers.
__global__ void __launch_bounds__(THREADS) chunk_sums_kernel(LinearChunksArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    bf16* k_tile = reinterpret_cast<bf16*>(raw);            // [64][DP]
    bf16* v_tile = k_tile + CHUNK * DP;                     // [64][EP]
    float* weight = reinterpret_cast<float*>(v_tile + CHUNK * EP);      // [64]
    const Chunk chunk(a, blockIdx.z, blockIdx.x);
    if (!chunk.live) return;
    const int head = a.head0 + blockIdx.y;
    load_rows<D>(k_tile, a.k + chunk.row * a.ldk + (long long)head * D, a.ldk, chunk.tokens);
    load_rows<E>(v_tile, a.v + chunk.row * a.ldv + (long long)head * E, a.ldv, chunk.tokens);
    copy_async_commit();
    if (threadIdx.x < CHUNK)
        weight[threadIdx.x] = threadIdx.x < chunk.tokens ? powf(a.decay[head], (float)(chunk.tokens - 1 - threadIdx.x)) : 0.f;
    copy_async_wait<0>();
    __syncthreads();
    constexpr int SPAN = 64, SPANS = (E + SPAN - 1) / SPAN;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int matrix = lane >> 3, within = lane & 7;
    float* sums = a.sums + ((long long)chunk.index * a.group + blockIdx.y) * D * E;
    for (int item = warp; item < D / 16 * SPANS; item += THREADS / 32) {
        const int m0 = item / SPANS * 16, n0 = item % SPANS * SPAN;
        float c[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) c[j][i] = 0.f;
#pragma unroll
        for (int kk = 0; kk < CHUNK / 16; ++kk) {
            unsigned keys[4], parts[3][4];
            // A operand, rows m0 .. m0 + 15 (of dim) by 16 tokens: matrices (rows, tokens), (rows + 8, tokens),
            // (rows, tokens + 8), (rows + 8, tokens + 8), each transposed on the way.
            ldmatrix_x4_trans(keys, k_tile + (kk * 16 + within + (matrix >> 1) * 8) * DP + m0 + (matrix & 1) * 8);
            const float2 w0 = *reinterpret_cast<const float2*>(weight + kk * 16 + 2 * t);
            const float2 w1 = *reinterpret_cast<const float2*>(weight + kk * 16 + 8 + 2 * t);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 key = unpack(keys[i]), w = i < 2 ? w0 : w1;
                split_pair(key.x * w.x, key.y * w.y, parts[0][i], parts[1][i], parts[2][i]);
            }
#pragma unroll
            for (int p = 0; p < 4; ++p) {                   // 16 columns at a time
                if (n0 + p * 16 >= E) continue;
                unsigned values[4];
                ldmatrix_x4_trans(values, v_tile + (kk * 16 + within + (matrix & 1) * 8) * EP + n0 + p * 16 + (matrix >> 1) * 8);
#pragma unroll
                for (int s = 2; s >= 0; --s) {              // the smallest part first
                    mma_bf16(c[2 * p], parts[s], values[0], values[1]);
                    mma_bf16(c[2 * p + 1], parts[s], values[2], values[3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int column = n0 + j * 8 + 2 * t;
            if (column >= E) continue;
            *reinterpret_cast<float2*>(sums + (long long)(m0 + g) * E + column) = make_float2(c[j][0], c[j][1]);
            *reinterpret_cast<float2*>(sums + (long long)(m0 + g + 8) * E + column) = make_float2(c[j][2], c[j][3]);
        }
    }
}

// ---------------------------------------------------------------- the states before the chunks
// A thread walks a sequence's chunks with four neighbouring elements of a head's state, a few chunks' sums in flight.
constexpr int WALK_THREADS = 128, AHEAD = 8;
__global__ void __launch_bounds__(WALK_THREADS) chunk_states_kernel(LinearChunksArgs a) {
    const int seq = blockIdx.z, head = a.head0 + blockIdx.y;
    const int row0 = a.seq_row0[seq], count = a.seq_len[seq];
    const long long at = 4 * ((long long)blockIdx.x * WALK_THREADS + threadIdx.x);
    if (count <= 0 || a.row_seq[row0] < 0 || at >= D * E) return;
    const int chunks = (count + CHUNK - 1) / CHUNK;
    const long long stride = (long long)a.group * D * E;
    const float* sums = a.sums + ((long long)first_chunk(row0, seq) * a.group + blockIdx.y) * D * E + at;
    bf16* before = a.before + 3 * (((long long)first_chunk(row0, seq) * a.group + blockIdx.y) * D * E) + at;
    float* kept = a.state + ((long long)a.seq_slot[seq] * a.heads + head) * D * E + at;
    const float decay = a.decay[head], keep = powf(decay, (float)CHUNK);
    float4 s = *reinterpret_cast<const float4*>(kept);
    float4 ahead[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (i < chunks) ahead[i] = *reinterpret_cast<const float4*>(sums + i * stride);
    for (int base = 0; base < chunks; base += AHEAD) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const int c = base + i;
            if (c < chunks) {
                const float4 sum = ahead[i];
                if (c + AHEAD < chunks) ahead[i] = *reinterpret_cast<const float4*>(sums + (c + AHEAD) * stride);
                uint2 parts[3];
                split_pair(s.x, s.y, parts[0].x, parts[1].x, parts[2].x);
                split_pair(s.z, s.w, parts[0].y, parts[1].y, parts[2].y);
#pragma unroll
                for (int p = 0; p < 3; ++p) *reinterpret_cast<uint2*>(before + 3 * c * stride + p * (D * E)) = parts[p];
                const float factor = c + 1 < chunks ? keep : powf(decay, (float)(count - c * CHUNK));
                s.x = fmaf(factor, s.x, sum.x); s.y = fmaf(factor, s.y, sum.y);
                s.z = fmaf(factor, s.z, sum.z); s.w = fmaf(factor, s.w, sum.w);
            }
        }
    }
    *reinterpret_cast<float4*>(kept) = s;
}

// ---------------------------------------------------------------- the read-out
// Four warps by 16 tokens, twice: of the pairs of 8-column tiles one half of the warps takes the even, the other the odd.
// First q S for the state before the chunk, slice by slice (SLICE rows of S in three parts), its rows times a^(i+1); then
// the scores q k^T, decayed and split in registers, times v into the same accumulators.
constexpr int PAIRS = E / 16, MINE = (PAIRS + 1) / 2;
constexpr size_t READ_SHARED = (size_t)(2 * CHUNK * DP + CHUNK * EP + 2 * 3 * SLICE * EP) * sizeof(bf16) + (CHUNK + 1) * sizeof(float);

__global__ void __launch_bounds__(THREADS) chunk_read_kernel(LinearChunksArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    bf16* q_tile = reinterpret_cast<bf16*>(raw);            // [64][DP]
    bf16* k_tile = q_tile + CHUNK * DP;                     // [64][DP]
    bf16* v_tile = k_tile + CHUNK * DP;                     // [64][EP]
    bf16* s_tile = v_tile + CHUNK * EP;                     // [2][3][SLICE][EP]
    float* power = reinterpret_cast<float*>(s_tile + 2 * 3 * SLICE * EP);       // [65]: a^0 .. a^64
    const Chunk chunk(a, blockIdx.z, blockIdx.x);
    if (!chunk.live) return;
    const int head = a.head0 + blockIdx.y;
    const bf16* before = a.before + 3 * (((long long)chunk.index * a.group + blockIdx.y) * D * E);
    auto load_slice = [&](int slice) {
        constexpr int PIECES = E / 8;
        bf16* target = s_tile + (slice & 1) * (3 * SLICE * EP);
        for (int i = threadIdx.x; i < 3 * SLICE * PIECES; i += THREADS) {
            const int r = i / PIECES, c = i - r * PIECES;                  // r: part * SLICE + row
            const int part = r / SLICE, row = slice * SLICE + r - part * SLICE;
            copy_async_16(target + r * EP + c * 8, before + ((long long)part * D + row) * E + c * 8, true);
        }
        copy_async_commit();
    };
    load_rows<D>(q_tile, a.q + chunk.row * a.ldq + (long long)head * D, a.ldq, chunk.tokens);
    load_slice(0);
    load_rows<D>(k_tile, a.k + chunk.row * a.ldk + (long long)head * D, a.ldk, chunk.tokens);
    load_rows<E>(v_tile, a.v + chunk.row * a.ldv + (long long)head * E, a.ldv, chunk.tokens);
    if (SLICES == 1) copy_async_commit();
    for (int i = threadIdx.x; i <= CHUNK; i += THREADS) power[i] = powf(a.decay[head], (float)i);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int matrix = lane >> 3, within = lane & 7;
    const int row = (warp & 3) * 16, side = warp >> 2;      // the warp's 16 tokens; its pairs: side, side + 2, ..
    float o[2 * MINE][4];
#pragma unroll
    for (int j = 0; j < 2 * MINE; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
    for (int slice = 0; slice < SLICES; ++slice) {
        if (slice + 1 < SLICES) {
            load_slice(slice + 1);
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        const bf16* current = s_tile + (slice & 1) * (3 * SLICE * EP);
#pragma unroll
        for (int kk = 0; kk < SLICE / 16; ++kk) {
            unsigned q[4];
            ldmatrix_x4(q, q_tile + (row + within + (matrix & 1) * 8) * DP + slice * SLICE + kk * 16 + (matrix >> 1) * 8);
#pragma unroll
            for (int p = 0; p < MINE; ++p) {
                const int column = (side + 2 * p) * 16;
                if (column >= E) continue;
#pragma unroll
                for (int part = 2; part >= 0; --part) {
                    unsigned s[4];
                    ldmatrix_x4_trans(s, current + (part * SLICE + kk * 16 + within + (matrix & 1) * 8) * EP + column + (matrix >> 1) * 8);
                    mma_bf16(o[2 * p], q, s[0], s[1]);
                    mma_bf16(o[2 * p + 1], q, s[2], s[3]);
                }
            }
        }
        __syncthreads();                                    // the slice is read: its buffer takes the one after next
    }
    const float below = power[row + g + 1], above = power[row + g + 9];
#pragma unroll
    for (int j = 0; j < 2 * MINE; ++j) {
        o[j][0] *= below; o[j][1] *= below;
        o[j][2] *= above; o[j][3] *= above;
    }
    // Scores against 16 keys at a time, only tiles that hold a key at or before the warp's last token.
    for (int kt = 0; kt <= (warp & 3); ++kt) {
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
            unsigned q[4], k[4];
            ldmatrix_x4(q, q_tile + (row + within + (matrix & 1) * 8) * DP + kk * 16 + (matrix >> 1) * 8);
            ldmatrix_x4(k, k_tile + (kt * 16 + within + (matrix >> 1) * 8) * DP + kk * 16 + (matrix & 1) * 8);
            mma_bf16(s[0], q, k[0], k[1]);
            mma_bf16(s[1], q, k[2], k[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int back = row + g + (i >> 1) * 8 - (kt * 16 + j * 8 + 2 * t + (i & 1));
                s[j][i] = back >= 0 ? s[j][i] * power[back] : 0.f;
            }
        unsigned parts[3][4];
        split_pair(s[0][0], s[0][1], parts[0][0], parts[1][0], parts[2][0]);
        split_pair(s[0][2], s[0][3], parts[0][1], parts[1][1], parts[2][1]);
        split_pair(s[1][0], s[1][1], parts[0][2], parts[1][2], parts[2][2]);
        split_pair(s[1][2], s[1][3], parts[0][3], parts[1][3], parts[2][3]);
#pragma unroll
        for (int p = 0; p < MINE; ++p) {
            const int column = (side + 2 * p) * 16;
            if (column >= E) continue;
            unsigned v[4];
            ldmatrix_x4_trans(v, v_tile + (kt * 16 + within + (matrix & 1) * 8) * EP + column + (matrix >> 1) * 8);
#pragma unroll
            for (int part = 2; part >= 0; --part) {
                mma_bf16(o[2 * p], parts[part], v[0], v[1]);
                mma_bf16(o[2 * p + 1], parts[part], v[2], v[3]);
            }
        }
    }
    float* out = a.out + (long long)chunk.row * a.heads * E + (long long)head * E;
#pragma unroll
    for (int p = 0; p < MINE; ++p) {
        const int column = (side + 2 * p) * 16;
        if (column >= E) continue;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int c = column + j * 8 + 2 * t;
            if (row + g < chunk.tokens)
                *reinterpret_cast<float2*>(out + (long long)(row + g) * a.heads * E + c) = make_float2(o[2 * p + j][0], o[2 * p + j][1]);
            if (row + g + 8 < chunk.tokens)
                *reinterpret_cast<float2*>(out + (long long)(row + g + 8) * a.heads * E + c) = make_float2(o[2 * p + j][2], o[2 * p + j][3]);
        }
    }
}

constexpr size_t SUMS_SHARED = (size_t)CHUNK * (DP + EP) * sizeof(bf16) + CHUNK * sizeof(float);

}  // namespace

// Floats (32-bit elements) of scratch memory a launch over `group` heads needs: the sums, then the states in three parts.
KIDI_API long long kidi_linear_chunks_scratch(int rows, int seqs, int group) {
    if (rows < 0 || seqs < 0 || group < 1) return -1;
    const long long chunks = rows / CHUNK + seqs + 1;
    const long long sums = chunks * group * D * E;
    return sums + (sums * 3 + 1) / 2;
}

KIDI_API int kidi_linear_chunks(const LinearChunksArgs* args, cudaStream_t stream) {
    const LinearChunksArgs& a = *args;
    if (a.seqs <= 0 || a.max_chunks <= 0) return 0;
    if (a.heads <= 0 || a.seqs > 65535 || a.group < 1 || a.group > 65535 || a.head0 < 0 || a.head0 + a.group > a.heads ||
        (a.ldq & 7) || (a.ldk & 7) || (a.ldv & 7) || ((uintptr_t)a.q & 15) || ((uintptr_t)a.k & 15) || ((uintptr_t)a.v & 15) ||
        ((uintptr_t)a.state & 15) || ((uintptr_t)a.out & 15) || ((uintptr_t)a.sums & 15) || ((uintptr_t)a.before & 15))
        return KIDI_REFUSED_SIZE;
    cudaError_t status = cudaFuncSetAttribute(chunk_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SUMS_SHARED);
    if (status == cudaSuccess)
        status = cudaFuncSetAttribute(chunk_read_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)READ_SHARED);
    if (status != cudaSuccess) return (int)status;
    const dim3 grid(a.max_chunks, a.group, a.seqs);
    int launched = kidi_launch(chunk_sums_kernel, grid, THREADS, SUMS_SHARED, stream, a);
    if (launched) return launched;
    const dim3 walk((D * E / 4 + WALK_THREADS - 1) / WALK_THREADS, a.group, a.seqs);
    launched = kidi_launch(chunk_states_kernel, walk, WALK_THREADS, 0, stream, a);
    if (launched) return launched;
    return kidi_launch(chunk_read_kernel, grid, THREADS, READ_SHARED, stream, a);
}
