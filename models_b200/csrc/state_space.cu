// A state-space recurrence with one decay per head and token (Mamba-2's scalar form); ragged sequences, float state per sequence.
//
// Per head h with its float state S [state][vdim] (group c = h / (heads / groups)):
//   dt_t = softplus(dt_in_t + dt_bias_h);   S <- exp(decay_h * dt_t) S + dt_t B_t x_t^T        (decay_h = -exp(A_log_h), a number <= 0)
//   y_t = S^T C_t + D_h x_t
// x [heads * vdim], B [groups * state] and C [groups * state] are columns of one row per token (the convolved projections).
// Here: the token-by-token walk (decoding, short steps, 32-bit mode, any sizes), and the norm that follows the recurrence:
//   v = y * silu(z);   out = out_scale * v / sqrt(mean of v^2 over the part + eps) * gain, a row being cut into equal parts.
// Everything is float arithmetic.  The form for long steps is csrc/state_space_chunks.cu.
#include "common.cuh"

MB_DEFINE_LAST_ERROR()

namespace mb {

__device__ __forceinline__ float sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

struct SpaceShape {
    int heads, groups, state, vdim;
    int x_at, b_at, c_at;  // first columns of the row's parts
};

// grid (ceil(vdim / (16 * warps)), heads, sequences); block warps * 32.  A warp owns 16 columns of one head's state: lane =
// 4 * n_lane + p_lane, four neighbouring columns a lane (p_lane), the rows n = n_lane + 8 i of the state in registers
// (i < kPer, state <= 8 kPer).  The sum over n of a read-out meets by shuffles over the eight n_lanes; a warp waits for no other.
// The next token's rows are asked for while a token is worked on.
template <typename T, typename R, int kPer, bool kVec>
__global__ void space_walk_kernel(const R* __restrict__ rows, int row_stride, const T* __restrict__ dt_in, int dt_stride,
                                  const float* __restrict__ decay, const float* __restrict__ dt_bias, const float* __restrict__ skip,
                                  float* __restrict__ state, size_t state_stride, const int* __restrict__ slots, const int* __restrict__ cu_q,
                                  float* __restrict__ y, SpaceShape shape) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int p_lane = lane & 3, n_lane = lane >> 2;
    const int head = blockIdx.y, seq = blockIdx.z;
    const int first = cu_q[seq], count = cu_q[seq + 1] - first;
    const int N = shape.state, P = shape.vdim;
    const int col = (blockIdx.x * warps + warp) * 16 + p_lane * 4;
    if (count <= 0 || (blockIdx.x * warps + warp) * 16 >= P) return;  // (whole warps leave)
    const int group = head / (shape.heads / shape.groups);
    float* stored = state + (size_t)slots[seq] * state_stride + (size_t)head * N * P;
    float s[kPer][4];
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
        const int n = n_lane + 8 * i;
        s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        if (n < N) {
            if (kVec) {
                if (col < P) {
                    const float4 v = *reinterpret_cast<const float4*>(stored + (size_t)n * P + col);
                    s[i][0] = v.x, s[i][1] = v.y, s[i][2] = v.z, s[i][3] = v.w;
                }
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (col + j < P) s[i][j] = stored[(size_t)n * P + col + j];
            }
        }
    }
    const float head_decay = decay[head], head_dt = dt_bias[head], head_skip = skip[head];
    float b[kPer], c[kPer], x[4], dt_raw;
    auto fetch = [&](int t, float (&bb)[kPer], float (&cc)[kPer], float (&xx)[4], float& dd) {
        const R* row = rows + (size_t)(first + t) * row_stride;
#pragma unroll
        for (int i = 0; i < kPer; ++i) {
            const int n = n_lane + 8 * i;
            bb[i] = n < N ? Num<R>::load(row + shape.b_at + (size_t)group * N + n) : 0.0f;
            cc[i] = n < N ? Num<R>::load(row + shape.c_at + (size_t)group * N + n) : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) xx[j] = col + j < P ? Num<R>::load(row + shape.x_at + (size_t)head * P + col + j) : 0.0f;
        dd = Num<T>::load(dt_in + (size_t)(first + t) * dt_stride + head);
    };
    fetch(0, b, c, x, dt_raw);
    for (int t = 0; t < count; ++t) {
        float b_next[kPer], c_next[kPer], x_next[4], dt_next;
        fetch(t + 1 < count ? t + 1 : t, b_next, c_next, x_next, dt_next);
        const float dt = softplus(dt_raw + head_dt);
        const float keep = expf(head_decay * dt);
        float write[4], sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int j = 0; j < 4; ++j) write[j] = dt * x[j];
#pragma unroll
        for (int i = 0; i < kPer; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                s[i][j] = fmaf(keep, s[i][j], b[i] * write[j]);
                sum[j] = fmaf(s[i][j], c[i], sum[j]);
            }
#pragma unroll
        for (int offset = 4; offset < 32; offset <<= 1)
#pragma unroll
            for (int j = 0; j < 4; ++j) sum[j] += __shfl_xor_sync(0xffffffffu, sum[j], offset);
        if (n_lane == 0) {
            float* dst = y + (size_t)(first + t) * shape.heads * P + (size_t)head * P + col;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (col + j < P) dst[j] = fmaf(head_skip, x[j], sum[j]);
        }
#pragma unroll
        for (int i = 0; i < kPer; ++i) b[i] = b_next[i], c[i] = c_next[i];
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = x_next[j];
        dt_raw = dt_next;
    }
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
        const int n = n_lane + 8 * i;
        if (n < N) {
            if (kVec) {
                if (col < P) *reinterpret_cast<float4*>(stored + (size_t)n * P + col) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (col + j < P) stored[(size_t)n * P + col + j] = s[i][j];
            }
        }
    }
}

// grid (tokens, parts); block a multiple of 32.  kVec neighbouring numbers a thread and step (8: 16-byte loads of bfloat16 rows); the
// first kKept steps' products stay in registers between the sum and the store, parts larger than that are read twice.
template <typename T, int kVec>
__device__ __forceinline__ void load_some(const T* p, float (&v)[kVec]) {
    if constexpr (kVec == 8) {
        load8(p, v);
    } else {
#pragma unroll
        for (int j = 0; j < kVec; ++j) v[j] = Num<T>::load(p + j);
    }
}

template <typename T, typename Y, int kVec, int kKept>
__global__ void __launch_bounds__(256)
gate_part_norm_kernel(const Y* __restrict__ y, const T* __restrict__ z, int z_stride, const float* __restrict__ gain, float eps,
                      T* __restrict__ out, int out_stride, float out_scale, int width, int size) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float scratch[32];
    const size_t token = blockIdx.x;
    const int at = blockIdx.y * size, step = blockDim.x * kVec;
    const Y* y_part = y + token * width + at;
    const T* z_part = z + token * z_stride + at;
    float kept[kKept][kVec];
    float squares = 0.0f;
    auto gated = [&](int c, float (&v)[kVec]) {
        float g[kVec];
        load_some<Y, kVec>(y_part + c, v);
        load_some<T, kVec>(z_part + c, g);
#pragma unroll
        for (int j = 0; j < kVec; ++j) v[j] *= g[j] * sigmoid(g[j]);
    };
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        const int c = threadIdx.x * kVec + i * step;
        if (c < size) {
            gated(c, kept[i]);
#pragma unroll
            for (int j = 0; j < kVec; ++j) squares = fmaf(kept[i][j], kept[i][j], squares);
        }
    }
    for (int c = threadIdx.x * kVec + kKept * step; c < size; c += step) {
        float v[kVec];
        gated(c, v);
#pragma unroll
        for (int j = 0; j < kVec; ++j) squares = fmaf(v[j], v[j], squares);
    }
    const float factor = out_scale / sqrtf(block_sum(squares, scratch) / (float)size + eps);
    auto store = [&](int c, float (&v)[kVec]) {
        float w[kVec];
        load_some<float, kVec>(gain + at + c, w);
#pragma unroll
        for (int j = 0; j < kVec; ++j) v[j] *= factor * w[j];
        T* dst = out + token * out_stride + at + c;
        if constexpr (kVec == 8) {
            store8(dst, v);
        } else {
#pragma unroll
            for (int j = 0; j < kVec; ++j) Num<T>::store(dst + j, v[j]);
        }
    };
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        const int c = threadIdx.x * kVec + i * step;
        if (c < size) store(c, kept[i]);
    }
    for (int c = threadIdx.x * kVec + kKept * step; c < size; c += step) {
        float v[kVec];
        gated(c, v);
        store(c, v);
    }
}

template <typename T, typename R, int kPer>
int launch_walk(const void* rows, int row_stride, const void* dt_in, int dt_stride, const float* decay, const float* dt_bias, const float* skip,
                float* state, size_t state_stride, const int* slots, const int* cu_q, int sequences, float* y, SpaceShape shape,
                cudaStream_t stream) {
    const int tiles = (shape.vdim + 15) / 16;
    const int warps = 1;  // (warps do not wait for one another: a block each spreads a few heads over more multiprocessors)
    const dim3 grid((tiles + warps - 1) / warps, shape.heads, sequences);
    const bool vec = shape.vdim % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
    if (vec)
        MB_LAUNCH("state_space_walk", (space_walk_kernel<T, R, kPer, true>), grid, dim3(32 * warps), 0, stream, true, (const R*)rows, row_stride,
                  (const T*)dt_in, dt_stride, decay, dt_bias, skip, state, state_stride, slots, cu_q, y, shape);
    else
        MB_LAUNCH("state_space_walk", (space_walk_kernel<T, R, kPer, false>), grid, dim3(32 * warps), 0, stream, true, (const R*)rows, row_stride,
                  (const T*)dt_in, dt_stride, decay, dt_bias, skip, state, state_stride, slots, cu_q, y, shape);
    return 0;
}

template <typename T, typename R, typename... Args>
int pick_walk(int state, Args... args) {
    if (state <= 16) return launch_walk<T, R, 2>(args...);
    if (state <= 32) return launch_walk<T, R, 4>(args...);
    if (state <= 64) return launch_walk<T, R, 8>(args...);
    if (state <= 128) return launch_walk<T, R, 16>(args...);
    if (state <= 256) return launch_walk<T, R, 32>(args...);
    if (state <= 512) return launch_walk<T, R, 64>(args...);  // (the registers overflow into local memory: correct, not fast)
    return fail("state_space_walk: a state of %d rows per head exceeds 512", state);
}

template <typename T, typename Y>
int gate_part_norm(const void* y, const void* z, int z_stride, const float* gain, float eps, void* out, int out_stride, float out_scale,
                   int tokens, int width, int parts, cudaStream_t stream) {
    const int size = width / parts;
    const uintptr_t starts = (uintptr_t)y | (uintptr_t)z | (uintptr_t)gain | (uintptr_t)out;
    const bool eight = size % 8 == 0 && width % 8 == 0 && !(starts & 15) && ((size_t)z_stride * sizeof(T)) % 16 == 0 && ((size_t)out_stride * sizeof(T)) % 16 == 0;
    const int vec = eight ? 8 : 1;
    int threads = 32;
    while (threads < 256 && threads * vec < size) threads *= 2;
#define MB_PART(VEC, KEPT)                                                                                                               \
    MB_LAUNCH("gate_part_norm", (gate_part_norm_kernel<T, Y, VEC, KEPT>), dim3(tokens, parts), dim3(threads), 0, stream, true, (const Y*)y, \
              (const T*)z, z_stride, gain, eps, (T*)out, out_stride, out_scale, width, size)
    if (eight && size <= threads * 8) MB_PART(8, 1);
    else if (eight) MB_PART(8, 4);
    else MB_PART(1, 8);
#undef MB_PART
    return 0;
}

}  // namespace mb

using namespace mb;

// rows (dtype row_dtype, row stride in elements): x from column x_at, B from b_at, C from c_at.  dt_in [tokens, heads] (dtype, row
// stride); decay (= -exp(A_log)), dt_bias, skip (D) [heads] float; state + slots[seq] * state_stride is [heads][state][vdim]
// floats, updated in place; y float [tokens][heads * vdim].
MB_EXPORT int mb_state_space_walk(const void* rows, int row_stride, int row_dtype, const void* dt_in, int dt_stride, int dtype, const float* decay,
                                  const float* dt_bias, const float* skip, float* state, size_t state_stride, const int* slots,
                                  const int* cu_q, int sequences, float* y, int heads, int groups, int state_rows, int vdim, int x_at,
                                  int b_at, int c_at, cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (heads <= 0 || groups <= 0 || heads % groups || state_rows <= 0 || vdim <= 0)
        return fail("state_space_walk: %d heads in %d groups, state %d x %d", heads, groups, state_rows, vdim);
    if (sequences > 65535 || heads > 65535) return fail("state_space_walk: %d sequences or %d heads exceed the grid limit 65535", sequences, heads);
    const SpaceShape shape{heads, groups, state_rows, vdim, x_at, b_at, c_at};
    int status;
#define MB_WALK(T, R) pick_walk<T, R>(state_rows, rows, row_stride, dt_in, dt_stride, decay, dt_bias, skip, state, state_stride, slots, cu_q, sequences, y, shape, stream)
    if (dtype == MB_F32 && row_dtype == MB_F32) status = MB_WALK(float, float);
    else if (dtype == MB_BF16 && row_dtype == MB_F32) status = MB_WALK(__nv_bfloat16, float);
    else return fail("state_space_walk: dtype codes %d and %d are not built together", dtype, row_dtype);
#undef MB_WALK
    return status ? status : check_launch("state_space_walk");
}

// y [tokens][width] (y_dtype, contiguous), z and out rows of one storage type (strides in elements), gain [width] float; `parts`
// equal parts of a row are normalised on their own.
MB_EXPORT int mb_gate_part_norm(const void* y, int y_dtype, const void* z, int z_stride, const float* gain, float eps, void* out, int out_stride,
                                int dtype, float out_scale, int tokens, int width, int parts, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (parts <= 0 || width <= 0 || width % parts || parts > 65535) return fail("gate_part_norm: %d numbers in %d parts", width, parts);
    int status;
#define MB_NORM(T, Y) gate_part_norm<T, Y>(y, z, z_stride, gain, eps, out, out_stride, out_scale, tokens, width, parts, stream)
    if (dtype == MB_F32 && y_dtype == MB_F32) status = MB_NORM(float, float);
    else if (dtype == MB_BF16 && y_dtype == MB_F32) status = MB_NORM(__nv_bfloat16, float);
    else if (dtype == MB_BF16 && y_dtype == MB_BF16) status = MB_NORM(__nv_bfloat16, __nv_bfloat16);
    else return fail("gate_part_norm: dtype codes %d and %d are not built together", dtype, y_dtype);
#undef MB_NORM
    return status ? status : check_launch("gate_part_norm");
}
