// The state-space recurrence of csrc/state_space.cu over long steps: bfloat16 storage, head sizes fixed at compile time
// (-DMB_STATE=N rows of the state, -DMB_VALUE_DIM=P columns: multiples of 16, N up to 256, P up to 128).
//
// The recurrence S_t = exp(a_t) S_(t-1) + dt_t B_t x_t^T, a_t = decay_h dt_t, y_t = S_t^T C_t + D_h x_t is linear in S with a number
// as coefficient, so a sequence's step is cut into chunks of 128 tokens.  With c_t the sum of a from the chunk's start up to t:
//   chunk_states:  W = sum_j exp(c_last - c_j) dt_j B_j x_j^T             what the chunk adds to the state         (all chunks at once)
//   carry_states:  S <- exp(c_last) S + W from chunk to chunk, leaving every chunk's starting state                (element by element)
//   chunk_outputs: y_i = exp(c_i) S_start^T C_i + sum_(j <= i) exp(c_i - c_j) dt_j (C_i . B_j) x_j + D x_i           (all chunks at once)
// The products run on the tensor cores.  B, C and x are bfloat16 numbers; what the design keeps in 32 bits -- decays, step sizes,
// the state, and everything multiplied by them -- enters a product as TWO bfloat16 numbers, its rounding and the rounding of the
// rest, with float sums.  Chunks are counted from the step's first token of the sequence; their slots in the scratch memory are
// cu_q[seq] / 128 + seq + chunk, which no two chunks share.
#include "common.cuh"

#if !defined(MB_STATE) || !defined(MB_VALUE_DIM)
#error "compile with -DMB_STATE=<rows of the state> -DMB_VALUE_DIM=<columns>"
#endif

MB_DEFINE_LAST_ERROR()

namespace mb {

using bf16 = __nv_bfloat16;
constexpr int N = MB_STATE, P = MB_VALUE_DIM, L = 128;
static_assert(N % 16 == 0 && N >= 16 && N <= 256, "the state's rows must be a multiple of 16 in 16..256");
static_assert(P % 16 == 0 && P >= 16 && P <= 128, "the state's columns must be a multiple of 16 in 16..128");
constexpr int kThreads = 256;
constexpr int kStateRow = N * 2 + 16, kValueRow = P * 2 + 16;  // padded shared-memory rows: ldmatrix reads without bank conflicts
constexpr int kNSteps = N / 16;
constexpr bool kKeepC = N <= 128;  // C fragments in registers; beyond that they are read again per use
// chunk_outputs: C rows, then one region that holds the starting state's two planes first and the B and x rows afterwards
constexpr int kStatePlanes = 2 * N * kValueRow, kRows = L * kStateRow + L * kValueRow;
constexpr int kRegion = kStatePlanes > kRows ? kStatePlanes : kRows;
constexpr bool kApart = L * kStateRow + kStatePlanes + kRows <= 112 * 1024;  // both fit beside each other with two blocks per multiprocessor
constexpr size_t kOutputBytes = (size_t)L * kStateRow + (kApart ? kStatePlanes + kRows : kRegion);
constexpr size_t kStatesBytes = (size_t)L * kStateRow + 2 * (size_t)L * kValueRow;

__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int kLeft>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(kLeft) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as a pair of bfloat16 roundings and the pair of what the roundings left over.
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 back = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - back.x, b - back.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct ChunkShape {
    int heads, groups;
    int x_at, b_at, c_at;  // first columns of the row's parts
};

// `rows` rows of kCols numbers (row stride in elements) from a step's token on into padded rows; rows beyond `valid` become zeros.
template <int kCols, int kRow>
__device__ __forceinline__ void load_rows(unsigned char* dst, const bf16* __restrict__ src, size_t stride, int rows, int valid) {
    constexpr int kPieces = kCols / 8;
    const uint32_t base = smem_u32(dst);
    for (int i = threadIdx.x; i < rows * kPieces; i += kThreads) {
        const int row = i / kPieces, piece = i % kPieces;
        if (row < valid)
            cp_async16(base + row * kRow + piece * 16, src + (size_t)row * stride + piece * 8);
        else
            *reinterpret_cast<uint4*>(dst + row * kRow + piece * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// dt and the running sums of decay * dt of the chunk's tokens into shared memory (tokens beyond `valid`: dt 0).  All threads.
__device__ __forceinline__ void chunk_decays(const bf16* __restrict__ dt_in, int dt_stride, float head_decay, float head_dt, int valid,
                                             float* dt_s, float* sum_s, float* warp_sums) {
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    float dt = 0.0f, a = 0.0f;
    if (t < L) {
        if (t < valid) dt = softplus(__bfloat162float(dt_in[(size_t)t * dt_stride]) + head_dt);
        a = head_decay * dt;
#pragma unroll
        for (int offset = 1; offset < 32; offset <<= 1) {
            const float before = __shfl_up_sync(0xffffffffu, a, offset);
            if (lane >= offset) a += before;
        }
        if (lane == 31) warp_sums[warp] = a;
    }
    __syncthreads();
    if (t < L) {
        for (int w = 0; w < warp; ++w) a += warp_sums[w];
        dt_s[t] = dt;
        sum_s[t] = a;
    }
    __syncthreads();
}

// grid (chunks of the longest sequence, heads, sequences); block 256.  added [slot][head][N][P] float, chunk_decay [slot][head] = exp(c_last).
__global__ void __launch_bounds__(kThreads)
chunk_states_kernel(const bf16* __restrict__ rows, int row_stride, const bf16* __restrict__ dt_in, int dt_stride, const float* __restrict__ decay,
                    const float* __restrict__ dt_bias, const int* __restrict__ cu_q, float* __restrict__ added, float* __restrict__ chunk_decay,
                    ChunkShape shape) {
    grid_launch_dependents();
    grid_dependency_wait();
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float dt_s[L], sum_s[L], warp_sums[8];
    const int seq = blockIdx.z, head = blockIdx.y, chunk = blockIdx.x;
    const int first = cu_q[seq], count = cu_q[seq + 1] - first;
    const int t0 = chunk * L;
    if (t0 >= count) return;
    const int valid = min(L, count - t0);
    const int group = head / (shape.heads / shape.groups);
    const size_t slot = (size_t)(first / L + seq + chunk);
    unsigned char* b_rows = smem;                       // [L][N]
    unsigned char* hi_rows = smem + L * kStateRow;      // [L][P]: x times its weight, rounding
    unsigned char* lo_rows = hi_rows + L * kValueRow;   // and rest
    const bf16* row0 = rows + (size_t)(first + t0) * row_stride;
    load_rows<N, kStateRow>(b_rows, row0 + shape.b_at + (size_t)group * N, row_stride, L, valid);
    cp_async_commit();
    chunk_decays(dt_in + (size_t)(first + t0) * dt_stride + head, dt_stride, decay[head], dt_bias[head], valid, dt_s, sum_s, warp_sums);
    const float last = sum_s[L - 1];
    if (threadIdx.x == 0) chunk_decay[slot * shape.heads + head] = expf(last);
    constexpr int kPieces = P / 8;
    for (int i = threadIdx.x; i < L * kPieces; i += kThreads) {
        const int row = i / kPieces, piece = i % kPieces;
        float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
        if (row < valid) load8(row0 + (size_t)row * row_stride + shape.x_at + (size_t)head * P + piece * 8, v);
        const float w = expf(last - sum_s[row]) * dt_s[row];
        uint4 hi, lo;
        split_pair(v[0] * w, v[1] * w, hi.x, lo.x);
        split_pair(v[2] * w, v[3] * w, hi.y, lo.y);
        split_pair(v[4] * w, v[5] * w, hi.z, lo.z);
        split_pair(v[6] * w, v[7] * w, hi.w, lo.w);
        *reinterpret_cast<uint4*>(hi_rows + row * kValueRow + piece * 16) = hi;
        *reinterpret_cast<uint4*>(lo_rows + row * kValueRow + piece * 16) = lo;
    }
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, group_id = lane >> 2, tid4 = lane & 3;
    const uint32_t b_base = smem_u32(b_rows), hi_base = smem_u32(hi_rows), lo_base = smem_u32(lo_rows);
    const int steps = (valid + 15) / 16;
    for (int tile = warp; tile < kNSteps; tile += kThreads / 32) {  // 16 rows of the state
        float acc[P / 8][4];
#pragma unroll
        for (int i = 0; i < P / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
        for (int ks = 0; ks < steps; ++ks) {
            uint32_t a[4];  // B transposed: rows of the operand are the state's rows, its k the tokens
            ldmatrix_x4_trans(a, b_base + (ks * 16 + (lane & 7) + (lane >> 4) * 8) * kStateRow + tile * 32 + ((lane >> 3) & 1) * 16);
            const uint32_t at = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kValueRow + (lane >> 4) * 16;
#pragma unroll
            for (int dp = 0; dp < P / 16; ++dp) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, hi_base + at + dp * 32);
                mma_bf16(acc[2 * dp], a, b[0], b[1]);
                mma_bf16(acc[2 * dp + 1], a, b[2], b[3]);
                ldmatrix_x4_trans(b, lo_base + at + dp * 32);
                mma_bf16(acc[2 * dp], a, b[0], b[1]);
                mma_bf16(acc[2 * dp + 1], a, b[2], b[3]);
            }
        }
        float* dst = added + ((slot * shape.heads + head) * N + tile * 16 + group_id) * (size_t)P + tid4 * 2;
#pragma unroll
        for (int i = 0; i < P / 8; ++i) {
            *reinterpret_cast<float2*>(dst + i * 8) = make_float2(acc[i][0], acc[i][1]);
            *reinterpret_cast<float2*>(dst + 8 * P + i * 8) = make_float2(acc[i][2], acc[i][3]);
        }
    }
}

// grid (N * P / 4 / 128, heads, sequences); block 128: four neighbouring elements of a head's state a thread, over all chunks.
__global__ void __launch_bounds__(128)
carry_states_kernel(const float* __restrict__ added, const float* __restrict__ chunk_decay, bf16* __restrict__ start_hi, bf16* __restrict__ start_lo,
                    float* __restrict__ state, size_t state_stride, const int* __restrict__ slots, const int* __restrict__ cu_q, int heads,
                    int aligned) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int seq = blockIdx.z, head = blockIdx.y, e = (blockIdx.x * 128 + threadIdx.x) * 4;
    const int first = cu_q[seq], count = cu_q[seq + 1] - first;
    if (count <= 0 || e >= N * P) return;
    const int chunks = (count + L - 1) / L;
    const size_t slot0 = (size_t)(first / L + seq);
    float* stored = state + (size_t)slots[seq] * state_stride + (size_t)head * N * P + e;
    float s[4];
    if (aligned) {
        const float4 v = *reinterpret_cast<const float4*>(stored);
        s[0] = v.x, s[1] = v.y, s[2] = v.z, s[3] = v.w;
    } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) s[j] = stored[j];
    }
    constexpr int kAhead = 4;
    for (int c0 = 0; c0 < chunks; c0 += kAhead) {
        float4 w[kAhead];
        float keep[kAhead];
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {  // (what a few chunks add is asked for before the first is used)
            const size_t at = (slot0 + min(c0 + u, chunks - 1)) * heads + head;
            w[u] = *reinterpret_cast<const float4*>(added + at * (N * P) + e);
            keep[u] = chunk_decay[at];
        }
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
            if (c0 + u >= chunks) break;
            const size_t at = ((slot0 + c0 + u) * heads + head) * (size_t)(N * P) + e;
            uint2 hi, lo;
            split_pair(s[0], s[1], hi.x, lo.x);
            split_pair(s[2], s[3], hi.y, lo.y);
            *reinterpret_cast<uint2*>(start_hi + at) = hi;
            *reinterpret_cast<uint2*>(start_lo + at) = lo;
            s[0] = fmaf(keep[u], s[0], w[u].x), s[1] = fmaf(keep[u], s[1], w[u].y);
            s[2] = fmaf(keep[u], s[2], w[u].z), s[3] = fmaf(keep[u], s[3], w[u].w);
        }
    }
    if (aligned) {
        *reinterpret_cast<float4*>(stored) = make_float4(s[0], s[1], s[2], s[3]);
    } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) stored[j] = s[j];
    }
}

// grid (chunks, heads, sequences); block 256: warp w owns the chunk's tokens 16 w .. 16 w + 15.
__global__ void __launch_bounds__(kThreads)
chunk_outputs_kernel(const bf16* __restrict__ rows, int row_stride, const bf16* __restrict__ dt_in, int dt_stride, const float* __restrict__ decay,
                     const float* __restrict__ dt_bias, const float* __restrict__ skip, const int* __restrict__ cu_q,
                     const bf16* __restrict__ start_hi, const bf16* __restrict__ start_lo, bf16* __restrict__ y, ChunkShape shape) {
    grid_launch_dependents();
    grid_dependency_wait();
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float dt_s[L], sum_s[L], warp_sums[8];
    const int seq = blockIdx.z, head = blockIdx.y, chunk = blockIdx.x;
    const int first = cu_q[seq], count = cu_q[seq + 1] - first;
    const int t0 = chunk * L;
    if (t0 >= count) return;
    const int valid = min(L, count - t0);
    const int group = head / (shape.heads / shape.groups);
    const size_t slot = (size_t)(first / L + seq + chunk);
    unsigned char* c_rows = smem;  // [L][N]
    unsigned char* planes = smem + L * kStateRow;
    unsigned char* b_rows = planes + (kApart ? kStatePlanes : 0);
    unsigned char* x_rows = b_rows + L * kStateRow;
    const bf16* row0 = rows + (size_t)(first + t0) * row_stride;
    load_rows<N, kStateRow>(c_rows, row0 + shape.c_at + (size_t)group * N, row_stride, L, valid);
    const size_t start_at = (slot * shape.heads + head) * (size_t)(N * P);
    load_rows<P, kValueRow>(planes, start_hi + start_at, P, N, N);
    load_rows<P, kValueRow>(planes + N * kValueRow, start_lo + start_at, P, N, N);
    cp_async_commit();
    auto load_bx = [&]() {
        load_rows<N, kStateRow>(b_rows, row0 + shape.b_at + (size_t)group * N, row_stride, L, valid);
        load_rows<P, kValueRow>(x_rows, row0 + shape.x_at + (size_t)head * P, row_stride, L, valid);
        cp_async_commit();
    };
    if (kApart) load_bx();
    chunk_decays(dt_in + (size_t)(first + t0) * dt_stride + head, dt_stride, decay[head], dt_bias[head], valid, dt_s, sum_s, warp_sums);
    if (kApart) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, group_id = lane >> 2, tid4 = lane & 3;
    const bool has_rows = warp * 16 < valid;
    const uint32_t c_base = smem_u32(c_rows) + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kStateRow + (lane >> 4) * 16;
    const uint32_t value_lane = ((lane & 7) + ((lane >> 3) & 1) * 8) * kValueRow + (lane >> 4) * 16;
    uint32_t c_kept[kKeepC ? kNSteps : 1][4];
    float o[P / 8][4];
#pragma unroll
    for (int i = 0; i < P / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float sums[2] = {0.0f, 0.0f};  // c_i of the warp's two rows of this lane
    if (has_rows) {
        const uint32_t hi_base = smem_u32(planes) + value_lane, lo_base = hi_base + N * kValueRow;
#pragma unroll
        for (int ks = 0; ks < kNSteps; ++ks) {
            uint32_t now[4];
            ldmatrix_x4(kKeepC ? c_kept[kKeepC ? ks : 0] : now, c_base + ks * 32);
            const uint32_t(&a)[4] = kKeepC ? c_kept[kKeepC ? ks : 0] : now;
#pragma unroll
            for (int dp = 0; dp < P / 16; ++dp) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, hi_base + ks * 16 * kValueRow + dp * 32);
                mma_bf16(o[2 * dp], a, b[0], b[1]);
                mma_bf16(o[2 * dp + 1], a, b[2], b[3]);
                ldmatrix_x4_trans(b, lo_base + ks * 16 * kValueRow + dp * 32);
                mma_bf16(o[2 * dp], a, b[0], b[1]);
                mma_bf16(o[2 * dp + 1], a, b[2], b[3]);
            }
        }
        sums[0] = sum_s[warp * 16 + group_id], sums[1] = sum_s[warp * 16 + group_id + 8];
        const float start_keep[2] = {expf(sums[0]), expf(sums[1])};
#pragma unroll
        for (int i = 0; i < P / 8; ++i) o[i][0] *= start_keep[0], o[i][1] *= start_keep[0], o[i][2] *= start_keep[1], o[i][3] *= start_keep[1];
    }
    if (!kApart) {
        __syncthreads();  // every warp is done with the planes
        load_bx();
    }
    cp_async_wait<0>();
    __syncthreads();
    if (!has_rows) return;
    const uint32_t b_base = smem_u32(b_rows), x_base = smem_u32(x_rows) + value_lane;
    for (int part = 0; part <= warp; ++part) {  // 16 earlier tokens at a time
        float s[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
        const uint32_t key = b_base + (part * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * kStateRow + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int ks = 0; ks < kNSteps; ++ks) {
            uint32_t now[4], b[4];
            if (!kKeepC) ldmatrix_x4(now, c_base + ks * 32);
            ldmatrix_x4(b, key + ks * 32);
            mma_bf16(s[0], kKeepC ? c_kept[kKeepC ? ks : 0] : now, b[0], b[1]);
            mma_bf16(s[1], kKeepC ? c_kept[kKeepC ? ks : 0] : now, b[2], b[3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int j = part * 16 + half * 8 + tid4 * 2 + (i & 1), row = warp * 16 + group_id + (i >> 1) * 8;
                s[half][i] = j <= row ? s[half][i] * (expf(sums[i >> 1] - sum_s[j]) * dt_s[j]) : 0.0f;
            }
        uint32_t hi[4], lo[4];
        split_pair(s[0][0], s[0][1], hi[0], lo[0]);
        split_pair(s[0][2], s[0][3], hi[1], lo[1]);
        split_pair(s[1][0], s[1][1], hi[2], lo[2]);
        split_pair(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
        for (int dp = 0; dp < P / 16; ++dp) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, x_base + part * 16 * kValueRow + dp * 32);
            mma_bf16(o[2 * dp], hi, b[0], b[1]);
            mma_bf16(o[2 * dp + 1], hi, b[2], b[3]);
            mma_bf16(o[2 * dp], lo, b[0], b[1]);
            mma_bf16(o[2 * dp + 1], lo, b[2], b[3]);
        }
    }
    const float head_skip = skip[head];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = warp * 16 + group_id + 8 * r;
        if (row >= valid) continue;
        bf16* dst = y + ((size_t)(first + t0 + row) * shape.heads + head) * P + tid4 * 2;
        const unsigned char* x_row = x_rows + row * kValueRow + tid4 * 4;
#pragma unroll
        for (int i = 0; i < P / 8; ++i) {
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x_row + i * 16));
            *reinterpret_cast<__nv_bfloat162*>(dst + i * 8) = __floats2bfloat162_rn(fmaf(head_skip, x.x, o[i][2 * r]), fmaf(head_skip, x.y, o[i][2 * r + 1]));
        }
    }
}

}  // namespace mb

using namespace mb;

MB_EXPORT int mb_state_space_chunk_tokens() { return L; }

// rows bfloat16 (row stride and part starts multiples of 8 elements, 16-byte aligned); dt_in bfloat16 [tokens, heads] (row stride);
// decay, dt_bias, skip [heads] float; state + slots[seq] * state_stride is [heads][N][P] floats, updated in place; y bfloat16
// [tokens][heads * P].  Scratch for `chunk_slots` >= tokens / 128 + sequences slots: added [slots][heads][N * P] float,
// start_hi and start_lo the same in bfloat16, chunk_decay [slots][heads] float.
MB_EXPORT int mb_state_space_chunks(const void* rows, int row_stride, const void* dt_in, int dt_stride, const float* decay, const float* dt_bias,
                                    const float* skip, float* state, size_t state_stride, const int* slots, const int* cu_q, int sequences,
                                    int max_q_len, void* y, float* added, void* start_hi, void* start_lo, float* chunk_decay, int heads, int groups,
                                    int x_at, int b_at, int c_at, cudaStream_t stream) {
    if (sequences <= 0 || max_q_len <= 0) return 0;
    if (heads <= 0 || groups <= 0 || heads % groups) return fail("state_space_chunks: %d heads in %d groups", heads, groups);
    if (sequences > 65535 || heads > 65535) return fail("state_space_chunks: %d sequences or %d heads exceed the grid limit 65535", sequences, heads);
    if (row_stride % 8 || x_at % 8 || b_at % 8 || c_at % 8 || ((uintptr_t)rows & 15)) return fail("state_space_chunks: rows must start on 16 bytes");
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(chunk_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kStatesBytes) != cudaSuccess ||
            cudaFuncSetAttribute(chunk_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kOutputBytes) != cudaSuccess)
            return fail("state_space_chunks: cannot reserve %zu bytes of shared memory", kOutputBytes);
        configured = true;
    }
    const ChunkShape shape{heads, groups, x_at, b_at, c_at};
    const dim3 grid((max_q_len + L - 1) / L, heads, sequences);
    const int aligned = state_stride % 4 == 0 && !((uintptr_t)state & 15) ? 1 : 0;
    MB_LAUNCH("state_space_chunks", chunk_states_kernel, grid, dim3(kThreads), kStatesBytes, stream, true, (const bf16*)rows, row_stride,
              (const bf16*)dt_in, dt_stride, decay, dt_bias, cu_q, added, chunk_decay, shape);
    MB_LAUNCH("state_space_chunks", carry_states_kernel, dim3((N * P / 4 + 127) / 128, heads, sequences), dim3(128), 0, stream, true, added,
              chunk_decay, (bf16*)start_hi, (bf16*)start_lo, state, state_stride, slots, cu_q, heads, aligned);
    MB_LAUNCH("state_space_chunks", chunk_outputs_kernel, grid, dim3(kThreads), kOutputBytes, stream, true, (const bf16*)rows, row_stride,
              (const bf16*)dt_in, dt_stride, decay, dt_bias, skip, cu_q, (const bf16*)start_hi, (const bf16*)start_lo, (bf16*)y, shape);
    return check_launch("state_space_chunks");
}
