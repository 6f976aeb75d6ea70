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
// With -DKIDI_LINEAR_WIDE=1 ("retention") q and k are turned by position and k is multiplied by a number, in 32-bit, on the
// way into the products: they are 32-bit numbers then and enter in three parts too (of a product of two such numbers the six
// partial products above 2^-24 are kept), and the read-out finishes a head: divided by its root mean square, times the SiLU
// or sigmoid of a gate, rounded to bfloat16.
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
    // the wide build only
    const float* cos_table; // [positions, rotary_dim / 2] or null: entries i and i + rotary_dim / 2 of a head's q and k turn
    const float* sin_table;
    const int* row_pos;     // [rows]
    int rotary_dim;
    float key_scale;
    const bf16* gate;       // [rows, ldg]: head h at h * vdim
    long long ldg;
    bf16* finished;         // [rows, ldf]: takes read / rms(read) * act(gate)
    long long ldf;
    float eps;
    int gate_silu;          // act: 1 SiLU, 0 sigmoid
};

namespace {

constexpr int D = KIDI_LINEAR_DIM, E = KIDI_LINEAR_VDIM;
static_assert(D % 16 == 0 && E % 16 == 0 && D >= 16 && E >= 16 && D <= 256 && E <= 256, "head widths: multiples of 16 up to 256");
constexpr int CHUNK = 64;
constexpr int THREADS = 256;
constexpr int DP = D + 8, EP = E + 8;               // row pitches: ldmatrix without bank conflicts
#ifndef KIDI_LINEAR_WIDE
#define KIDI_LINEAR_WIDE 0
#endif
constexpr bool WIDE = KIDI_LINEAR_WIDE != 0;
constexpr int SCORE_PITCH = CHUNK + 8;
// Shared memory of the wide read-out with slices of `slice` rows of the state: two regions, one for q in three parts and
// later the scores in three parts, one for the slices, then k in three parts, then v; the decay's powers and the rows' sums
// of squares. (Two blocks of head widths 128 x 128 fit an SM.)
__host__ __device__ constexpr size_t larger(size_t x, size_t y) { return x > y ? x : y; }
__host__ __device__ constexpr size_t wide_first_region() { return larger((size_t)3 * CHUNK * DP, (size_t)3 * CHUNK * SCORE_PITCH); }
__host__ __device__ constexpr size_t wide_second_region(int slice) {
    return larger(larger((size_t)2 * 3 * slice * EP, (size_t)3 * CHUNK * DP), (size_t)CHUNK * EP);
}
__host__ __device__ constexpr size_t wide_read_bytes(int slice) {
    return (wide_first_region() + wide_second_region(slice)) * sizeof(bf16) + (size_t)(CHUNK + 4 + 4 * CHUNK) * sizeof(float);
}
constexpr size_t MOST_SHARED = 227 * 1024;
static_assert(!WIDE || wide_read_bytes(16) <= MOST_SHARED, "head widths of the wide build: too large for shared memory");
constexpr int SLICE = D % 32 == 0 && (!WIDE || wide_read_bytes(32) <= MOST_SHARED) ? 32 : 16;   // rows of the state that are
                                                                                             // in shared memory at a time
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

// The wide build: a chunk's rows of q or k (COUNT tiles at once: they turn by the same angles) as 32-bit numbers, turned by
// position; `take(tile, row, column, x, y)` gets two neighbouring entries, or, where half the rotary width is odd,
// `take_one(tile, row, column, x)` every entry. A warp takes a row; a lane that takes entries of rotated pairs has read their
// partners before it hands any of them on.
template <int WARPS, int COUNT, typename Take, typename TakeOne>
__device__ __forceinline__ void widen(const bf16* const (&tiles)[COUNT], const LinearChunksArgs& a, int row0, int tokens,
                                      Take take, TakeOne take_one) {
    const int half = a.cos_table ? a.rotary_dim / 2 : 0, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int position0 = half ? a.row_pos[row0] : 0;            // a sequence's rows of a step follow one another
#pragma unroll 4
    for (int i = 0; i < CHUNK / WARPS; ++i) {
        const int r = warp + i * WARPS;
        const long long angles = (long long)(position0 + min(r, tokens - 1)) * half;
        if (half & 1) {
            for (int c = lane; c < D - half; c += 32) {          // pairs, then single entries
                const bool pair = c < half;
                const float cosine = pair ? a.cos_table[angles + c] : 1.f, sine = pair ? a.sin_table[angles + c] : 0.f;
#pragma unroll
                for (int tile = 0; tile < COUNT; ++tile) {
                    const bf16* source = tiles[tile] + r * DP;
                    const float u = pair ? to_float(source[c]) : 0.f, v = to_float(source[c + half]);
                    if (pair) take_one(tile, r, c, u * cosine - v * sine);
                    take_one(tile, r, c + half, pair ? v * cosine + u * sine : v);
                }
            }
            continue;
        }
        for (int c = 2 * lane; c < D - half; c += 64) {          // two pairs, then two single entries
            const bool pair = c < half;
            float2 cosine = make_float2(1.f, 1.f), sine = make_float2(0.f, 0.f);
            if (pair) {
                cosine = *reinterpret_cast<const float2*>(a.cos_table + angles + c);
                sine = *reinterpret_cast<const float2*>(a.sin_table + angles + c);
            }
#pragma unroll
            for (int tile = 0; tile < COUNT; ++tile) {
                const bf16* source = tiles[tile] + r * DP + c;
                const float2 v = unpack(*reinterpret_cast<const unsigned*>(source + half));
                if (pair) {
                    const float2 u = unpack(*reinterpret_cast<const unsigned*>(source));
                    take(tile, r, c, u.x * cosine.x - v.x * sine.x, u.y * cosine.y - v.y * sine.y);
                    take(tile, r, c + half, v.x * cosine.x + u.x * sine.x, v.y * cosine.y + u.y * sine.y);
                } else {
                    take(tile, r, c + half, v.x, v.y);
                }
            }
        }
    }
}

// ---------------------------------------------------------------- a chunk's own sum
// [dim, vdim] = sum over j of a^(n-1-j) k_j v_j^T. A warp takes 16 rows (of dim) by up to 64 columns (of vdim) at a time;
// the keys come transposed out of shared memory, are decayed and split in registers.
__global__ void __launch_bounds__(THREADS) chunk_sums_kernel(LinearChunksArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    bf16* k_tile = reinterpret_cast<bf16*>(raw);            // [64][DP]
    bf16* v_tile = k_tile + CHUNK * DP;                     // [64][EP]
    float* weight = reinterpret_cast<float*>(v_tile + CHUNK * EP);      // [64]
    float* wide_keys = weight + CHUNK;                      // the wide build: [64][D + 4]
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
    if constexpr (WIDE) {
        const bf16* const tiles[1] = {k_tile};
        widen<THREADS / 32>(tiles, a, chunk.row, chunk.tokens,
              [&](int, int r, int c, float x, float y) {
                  *reinterpret_cast<float2*>(wide_keys + r * (D + 4) + c) = make_float2(x * a.key_scale, y * a.key_scale);
              },
              [&](int, int r, int c, float x) { wide_keys[r * (D + 4) + c] = x * a.key_scale; });
        __syncthreads();
    }
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
            if constexpr (!WIDE)
                ldmatrix_x4_trans(keys, k_tile + (kk * 16 + within + (matrix >> 1) * 8) * DP + m0 + (matrix & 1) * 8);
            const float2 w0 = *reinterpret_cast<const float2*>(weight + kk * 16 + 2 * t);
            const float2 w1 = *reinterpret_cast<const float2*>(weight + kk * 16 + 8 + 2 * t);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                float2 key;
                if constexpr (WIDE) {                       // rows m0 + g (+ 8), tokens 2t, 2t + 1 (+ 8)
                    const float* from = wide_keys + (kk * 16 + 2 * t + (i >> 1) * 8) * (D + 4) + m0 + g + (i & 1) * 8;
                    key = make_float2(from[0], from[D + 4]);
                } else {
                    key = unpack(keys[i]);
                }
                const float2 w = i < 2 ? w0 : w1;
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
constexpr int PAIRS = E / 16;
#if !KIDI_LINEAR_WIDE
constexpr int MINE = (PAIRS + 1) / 2;
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

#else   // KIDI_LINEAR_WIDE
// ---------------------------------------------------------------- the read-out of the wide build
// Sixteen warps: four times 16 tokens by four sides (a side takes every fourth pair of 8-column tiles). q and k are widened
// and split in shared memory once; the scores of 16 tokens against 16 keys are one warp's (side = key tile), which leaves
// them, decayed and split, where q was.
constexpr int WIDE_THREADS = 512, SIDES = 4, WIDE_MINE = (PAIRS + SIDES - 1) / SIDES;

// Three parts of x, the largest first.
__device__ __forceinline__ void split_store(bf16* at, int plane, float x) {
    const bf16 first = __float2bfloat16_rn(x);
    x -= __bfloat162float(first);
    const bf16 second = __float2bfloat16_rn(x);
    at[0] = first;
    at[plane] = second;
    at[2 * plane] = __float2bfloat16_rn(x - __bfloat162float(second));
}

__global__ void __launch_bounds__(WIDE_THREADS, 2) chunk_read_wide_kernel(LinearChunksArgs a) {
    extern __shared__ __align__(16) unsigned char raw[];
    constexpr int PLANE = CHUNK * DP, SCORE_PLANE = CHUNK * SCORE_PITCH;
    bf16* q_parts = reinterpret_cast<bf16*>(raw);           // [3][64][DP] (the bfloat16 rows first stand in the first plane)
    bf16* score_parts = q_parts;                            // then [3][64][SCORE_PITCH]
    bf16* s_tile = q_parts + wide_first_region();           // [2][3][SLICE][EP]
    bf16* k_parts = s_tile;                                 // then [3][64][DP]
    bf16* v_tile = s_tile;                                  // then [64][EP]
    float* power = reinterpret_cast<float*>(s_tile + wide_second_region(SLICE));      // [65]: a^0 .. a^64
    float* squares = power + CHUNK + 4;                     // [SIDES][64]
    const Chunk chunk(a, blockIdx.z, blockIdx.x);
    if (!chunk.live) return;
    const int head = a.head0 + blockIdx.y;
    const bf16* before = a.before + 3 * (((long long)chunk.index * a.group + blockIdx.y) * D * E);
    auto load_rows_wide = [&](bf16* tile, const bf16* source, long long ld, int width, int pitch) {
        const int pieces = width / 8;
        for (int i = threadIdx.x; i < CHUNK * pieces; i += WIDE_THREADS) {
            const int r = i / pieces, c = i - r * pieces;
            const bool valid = r < chunk.tokens;
            copy_async_16(tile + r * pitch + c * 8, source + (long long)(valid ? r : 0) * ld + c * 8, valid);
        }
    };
    auto load_slice = [&](int slice) {
        constexpr int PIECES = E / 8;
        bf16* target = s_tile + (slice & 1) * (3 * SLICE * EP);
        for (int i = threadIdx.x; i < 3 * SLICE * PIECES; i += WIDE_THREADS) {
            const int r = i / PIECES, c = i - r * PIECES;                  // r: part * SLICE + row
            const int part = r / SLICE, row = slice * SLICE + r - part * SLICE;
            copy_async_16(target + r * EP + c * 8, before + ((long long)part * D + row) * E + c * 8, true);
        }
        copy_async_commit();
    };
    load_rows_wide(q_parts, a.q + chunk.row * a.ldq + (long long)head * D, a.ldq, D, DP);
    copy_async_commit();
    load_slice(0);
    for (int i = threadIdx.x; i <= CHUNK; i += WIDE_THREADS) power[i] = powf(a.decay[head], (float)i);
    copy_async_wait<1>();
    __syncthreads();
    // (In place: a thread reads an entry and its partner before it writes either, and nobody else reads them.)
    auto widen_in_place = [&](bf16* planes, float scale) {
        const bf16* const tiles[1] = {planes};
        widen<WIDE_THREADS / 32>(tiles, a, chunk.row, chunk.tokens,
              [&](int, int r, int c, float x, float y) {
                  unsigned parts[3];
                  split_pair(x * scale, y * scale, parts[0], parts[1], parts[2]);
#pragma unroll
                  for (int part = 0; part < 3; ++part) *reinterpret_cast<unsigned*>(planes + part * PLANE + r * DP + c) = parts[part];
              },
              [&](int, int r, int c, float x) { split_store(planes + r * DP + c, PLANE, x * scale); });
    };
    widen_in_place(q_parts, 1.f);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int matrix = lane >> 3, within = lane & 7;
    const int row = (warp & 3) * 16, side = warp >> 2;      // the warp's 16 tokens; its pairs: side, side + SIDES, ..
    float o[2 * WIDE_MINE][4];
#pragma unroll
    for (int j = 0; j < 2 * WIDE_MINE; ++j)
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
            unsigned q[3][4];
#pragma unroll
            for (int part = 0; part < 3; ++part)
                ldmatrix_x4(q[part], q_parts + part * PLANE + (row + within + (matrix & 1) * 8) * DP + slice * SLICE + kk * 16 + (matrix >> 1) * 8);
#pragma unroll
            for (int p = 0; p < WIDE_MINE; ++p) {
                const int column = (side + SIDES * p) * 16;
                if (column >= E) continue;
                unsigned s[3][4];
#pragma unroll
                for (int part = 0; part < 3; ++part)
                    ldmatrix_x4_trans(s[part], current + (part * SLICE + kk * 16 + within + (matrix & 1) * 8) * EP + column + (matrix >> 1) * 8);
#pragma unroll
                for (int order = 2; order >= 0; --order)    // the smallest partial products first
#pragma unroll
                    for (int part = order; part >= 0; --part) {
                        mma_bf16(o[2 * p], q[part], s[order - part][0], s[order - part][1]);
                        mma_bf16(o[2 * p + 1], q[part], s[order - part][2], s[order - part][3]);
                    }
            }
        }
        __syncthreads();                                    // the slice is read: its buffer takes the one after next
    }
    load_rows_wide(k_parts, a.k + chunk.row * a.ldk + (long long)head * D, a.ldk, D, DP);
    copy_async_commit();
    const float below = power[row + g + 1], above = power[row + g + 9];
#pragma unroll
    for (int j = 0; j < 2 * WIDE_MINE; ++j) {
        o[j][0] *= below; o[j][1] *= below;
        o[j][2] *= above; o[j][3] *= above;
    }
    // Scores: this warp's 16 tokens against key tile `side`, where it holds a key at or before the last of them.
    copy_async_wait<0>();
    __syncthreads();
    widen_in_place(k_parts, a.key_scale);
    __syncthreads();
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    if (side <= (warp & 3)) {
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
            unsigned q[3][4], k[3][4];
#pragma unroll
            for (int part = 0; part < 3; ++part) {
                ldmatrix_x4(q[part], q_parts + part * PLANE + (row + within + (matrix & 1) * 8) * DP + kk * 16 + (matrix >> 1) * 8);
                ldmatrix_x4(k[part], k_parts + part * PLANE + (side * 16 + within + (matrix >> 1) * 8) * DP + kk * 16 + (matrix & 1) * 8);
            }
#pragma unroll
            for (int order = 2; order >= 0; --order)
#pragma unroll
                for (int part = order; part >= 0; --part) {
                    mma_bf16(s[0], q[part], k[order - part][0], k[order - part][1]);
                    mma_bf16(s[1], q[part], k[order - part][2], k[order - part][3]);
                }
        }
    }
    __syncthreads();                                        // q and k are read: the scores and v take their places
    load_rows_wide(v_tile, a.v + chunk.row * a.ldv + (long long)head * E, a.ldv, E, EP);
    copy_async_commit();
    if (side <= (warp & 3)) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; i += 2) {
                const int r = row + g + (i >> 1) * 8, key = side * 16 + j * 8 + 2 * t, back = r - key;
                const float x = back >= 0 ? s[j][i] * power[back] : 0.f, y = back >= 1 ? s[j][i + 1] * power[back - 1] : 0.f;
                unsigned parts[3];
                split_pair(x, y, parts[0], parts[1], parts[2]);
#pragma unroll
                for (int part = 0; part < 3; ++part)
                    *reinterpret_cast<unsigned*>(score_parts + part * SCORE_PLANE + r * SCORE_PITCH + key) = parts[part];
            }
    }
    copy_async_wait<0>();
    __syncthreads();
    for (int kt = 0; kt <= (warp & 3); ++kt) {
        unsigned parts[3][4];
#pragma unroll
        for (int part = 0; part < 3; ++part)
            ldmatrix_x4(parts[part], score_parts + part * SCORE_PLANE + (row + within + (matrix & 1) * 8) * SCORE_PITCH + kt * 16 + (matrix >> 1) * 8);
#pragma unroll
        for (int p = 0; p < WIDE_MINE; ++p) {
            const int column = (side + SIDES * p) * 16;
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
    // The finish: a row's sum of squares over its columns (a quad's lanes, then the sides in order), norm, gate.
    float square[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 2 * WIDE_MINE; ++j)                 // (columns that do not exist hold zeros)
#pragma unroll
        for (int i = 0; i < 4; ++i) square[i >> 1] = fmaf(o[j][i], o[j][i], square[i >> 1]);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        square[i] += __shfl_xor_sync(0xffffffffu, square[i], 1);
        square[i] += __shfl_xor_sync(0xffffffffu, square[i], 2);
        if (t == 0) squares[side * CHUNK + row + g + i * 8] = square[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = row + g + i * 8;
        if (r >= chunk.tokens) continue;
        const float total = squares[r] + squares[CHUNK + r] + squares[2 * CHUNK + r] + squares[3 * CHUNK + r];
        const float inv = 1.0f / sqrtf(total / (float)E + a.eps);
        const bf16* gate = a.gate + (long long)(chunk.row + r) * a.ldg + (long long)head * E;
        bf16* out = a.finished + (long long)(chunk.row + r) * a.ldf + (long long)head * E;
#pragma unroll
        for (int p = 0; p < WIDE_MINE; ++p) {
            const int column = (side + SIDES * p) * 16;
            if (column >= E) continue;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int c = column + j * 8 + 2 * t;
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c));
                // (sigmoid with the fast exponential and division: the result is rounded to bfloat16)
                const float x = __fdividef(a.gate_silu ? z.x : 1.f, 1.0f + __expf(fminf(-z.x, 80.f)));
                const float y = __fdividef(a.gate_silu ? z.y : 1.f, 1.0f + __expf(fminf(-z.y, 80.f)));
                *reinterpret_cast<__nv_bfloat162*>(out + c) =
                    __floats2bfloat162_rn(o[2 * p + j][2 * i] * inv * x, o[2 * p + j][2 * i + 1] * inv * y);
            }
        }
    }
}

#endif  // KIDI_LINEAR_WIDE

constexpr size_t SUMS_SHARED = (size_t)CHUNK * (DP + EP) * sizeof(bf16) + (CHUNK + (WIDE ? CHUNK * (D + 4) : 0)) * sizeof(float);

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
#if KIDI_LINEAR_WIDE
    if (!a.row_pos || !a.gate || !a.finished || (a.ldg & 1) || (a.ldf & 1) || ((uintptr_t)a.gate & 3) ||
        ((uintptr_t)a.finished & 3) ||
        (a.cos_table && (!a.sin_table || a.rotary_dim < 0 || (a.rotary_dim & 1) || a.rotary_dim > D)))
        return KIDI_REFUSED_SIZE;
    const auto read_kernel = chunk_read_wide_kernel;
    const size_t read_shared = wide_read_bytes(SLICE);
    const int read_threads = WIDE_THREADS;
#else
    const auto read_kernel = chunk_read_kernel;
    const size_t read_shared = READ_SHARED;
    const int read_threads = THREADS;
#endif
    cudaError_t status = cudaFuncSetAttribute(chunk_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SUMS_SHARED);
    if (status == cudaSuccess)
        status = cudaFuncSetAttribute(read_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)read_shared);
    if (status != cudaSuccess) return (int)status;
    const dim3 grid(a.max_chunks, a.group, a.seqs);
    int launched = kidi_launch(chunk_sums_kernel, grid, THREADS, SUMS_SHARED, stream, a);
    if (launched) return launched;
    const dim3 walk((D * E / 4 + WALK_THREADS - 1) / WALK_THREADS, a.group, a.seqs);
    launched = kidi_launch(chunk_states_kernel, walk, WALK_THREADS, 0, stream, a);
    if (launched) return launched;
    return kidi_launch(read_kernel, grid, read_threads, read_shared, stream, a);
}
