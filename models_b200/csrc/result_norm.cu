// Norms on a sublayer's result on its way into the float residual stream, with the next reader's rows made on the way.
//
//   dynamic tanh:  N(v) = tanh(alpha * v) * weight + bias, element by element (alpha one number, no mean and no variance)
//   root mean square:  R(v) = v / sqrt(mean(v^2) + eps) * weight over a row
//
//   result_tanh_add:  x += N(y);      result_rms_add:  x += R(y)
//
// y is a row of float sums, or the equally weighted sum of a row's expert results (ExpertSum).  After the addition the new row of x
// may be left for its next reader in the storage type: as it is, or through that reader's own dynamic tanh (Then).  Everything
// is float arithmetic.  Beside them the dynamic tanh alone, and the product of a gate with a table row of the token
// (side_gate: out = gelu_tanh(gate) * table[token]).
#include "common.cuh"

MB_DEFINE_LAST_ERROR()

namespace mb {

struct Tanh {
    float alpha;
    const float* weight;
    const float* bias;
};

// What happens to the new row of x: kind 0 nothing, 1 stored as it is, 2 stored through a dynamic tanh.
struct Then {
    int kind;
    Tanh norm;
};

// y[t] = weight * sum over a token's `top` entries of slot_out[place(t * top + s)], place = position[.] or the entry itself.
struct ExpertSum {
    const int* position;
    int top;
    float weight;
};

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

__device__ __forceinline__ float tanh_norm(float v, const Tanh& n, int c) { return fmaf(tanhf(n.alpha * v), n.weight[c], n.bias[c]); }
__device__ __forceinline__ float4 tanh_norm4(float4 v, const Tanh& n, int c) {
    const float4 w = load4(n.weight + c), b = load4(n.bias + c);
    return make_float4(fmaf(tanhf(n.alpha * v.x), w.x, b.x), fmaf(tanhf(n.alpha * v.y), w.y, b.y), fmaf(tanhf(n.alpha * v.z), w.z, b.z),
                       fmaf(tanhf(n.alpha * v.w), w.w, b.w));
}

// grid (ceil(rows * width / kVec / 256)); block 256; kVec columns a thread.
template <typename T, int kVec>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows, Tanh norm, T* __restrict__ out, size_t total, int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int per = width / kVec, c = (int)(i % per) * kVec;
    const size_t r = i / per;
    const size_t row = rows != nullptr ? (size_t)rows[r] : r;
    if (kVec == 4)
        store4(out + r * width + c, tanh_norm4(load4(x + row * width + c), norm, c));
    else
        Num<T>::store(out + r * width + c, tanh_norm(x[row * width + c], norm, c));
}

template <typename T, int kVec>
__global__ void __launch_bounds__(256)
tanh_add_kernel(float* __restrict__ x, const float* __restrict__ y, ExpertSum sum, Tanh norm, Then then, T* __restrict__ out, size_t total,
                int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int per = width / kVec, c = (int)(i % per) * kVec;
    const size_t t = i / per, at = t * width + c;
    if (kVec == 4) {
        float4 v;
        if (sum.top == 0) {
            v = load4(y + at);
        } else {
            v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            for (int s = 0; s < sum.top; ++s) {
                const size_t entry = t * sum.top + s;
                const float4 e = load4(y + (sum.position != nullptr ? (size_t)sum.position[entry] : entry) * width + c);
                v.x = fmaf(sum.weight, e.x, v.x), v.y = fmaf(sum.weight, e.y, v.y);
                v.z = fmaf(sum.weight, e.z, v.z), v.w = fmaf(sum.weight, e.w, v.w);
            }
        }
        const float4 old = load4(x + at), n = tanh_norm4(v, norm, c);
        const float4 now = make_float4(old.x + n.x, old.y + n.y, old.z + n.z, old.w + n.w);
        store4(x + at, now);
        if (then.kind == 1) store4(out + at, now);
        if (then.kind == 2) store4(out + at, tanh_norm4(now, then.norm, c));
    } else {
        float v = 0.0f;
        if (sum.top == 0) {
            v = y[at];
        } else {
            for (int s = 0; s < sum.top; ++s) {
                const size_t entry = t * sum.top + s;
                v = fmaf(sum.weight, y[(sum.position != nullptr ? (size_t)sum.position[entry] : entry) * width + c], v);
            }
        }
        const float now = x[at] + tanh_norm(v, norm, c);
        x[at] = now;
        if (then.kind == 1) Num<T>::store(out + at, now);
        if (then.kind == 2) Num<T>::store(out + at, tanh_norm(now, then.norm, c));
    }
}

// grid (rows); block a multiple of 32.  x += y / sqrt(mean(y^2) + eps) * weight.  Rows of up to kKept * blockDim.x * kVec numbers
// stay in registers between the sum and the addition.
template <typename T, int kVec, int kKept>
__global__ void rms_add_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ weight, float eps, Then then,
                               T* __restrict__ out, int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float scratch[32];
    const size_t row = (size_t)blockIdx.x * width;
    const int step = blockDim.x * kVec;
    float kept[kKept][kVec], old[kKept][kVec];
    float squares = 0.0f;
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        const int c = threadIdx.x * kVec + i * step;
#pragma unroll
        for (int j = 0; j < kVec; ++j) kept[i][j] = old[i][j] = 0.0f;
        if (c < width) {
            if (kVec == 4) {
                const float4 a = load4(y + row + c), b = load4(x + row + c);
                kept[i][0] = a.x, kept[i][1 % kVec] = a.y, kept[i][2 % kVec] = a.z, kept[i][3 % kVec] = a.w;
                old[i][0] = b.x, old[i][1 % kVec] = b.y, old[i][2 % kVec] = b.z, old[i][3 % kVec] = b.w;
            } else {
                kept[i][0] = y[row + c];
                old[i][0] = x[row + c];
            }
        }
#pragma unroll
        for (int j = 0; j < kVec; ++j) squares = fmaf(kept[i][j], kept[i][j], squares);
    }
    const float factor = 1.0f / sqrtf(block_sum(squares, scratch) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < kKept; ++i) {
        const int c = threadIdx.x * kVec + i * step;
        if (c >= width) continue;
        if (kVec == 4) {
            const float4 w = load4(weight + c);
            const float4 now = make_float4(fmaf(kept[i][0] * factor, w.x, old[i][0]), fmaf(kept[i][1 % kVec] * factor, w.y, old[i][1 % kVec]),
                                           fmaf(kept[i][2 % kVec] * factor, w.z, old[i][2 % kVec]), fmaf(kept[i][3 % kVec] * factor, w.w, old[i][3 % kVec]));
            store4(x + row + c, now);
            if (then.kind == 1) store4(out + row + c, now);
            if (then.kind == 2) store4(out + row + c, tanh_norm4(now, then.norm, c));
        } else {
            const float now = fmaf(kept[i][0] * factor, weight[c], old[i][0]);
            x[row + c] = now;
            if (then.kind == 1) Num<T>::store(out + row + c, now);
            if (then.kind == 2) Num<T>::store(out + row + c, tanh_norm(now, then.norm, c));
        }
    }
}

// out[t, c] = gelu_tanh(gate[t, c]) * table[token[t], c] for c < dim, 0 for dim <= c < columns.
template <typename T>
__global__ void __launch_bounds__(256)
side_gate_kernel(const float* __restrict__ gate, int gate_stride, const T* __restrict__ table, const int* __restrict__ tokens, int dim,
                 T* __restrict__ out, int columns, size_t total) {
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / columns;
    const int c = (int)(i % columns);
    float v = 0.0f;
    if (c < dim) v = gate_activation(MB_ACT_GELU_TANH, gate[t * gate_stride + c]) * Num<T>::load(table + (size_t)tokens[t] * dim + c);
    Num<T>::store(out + i, v);
}

inline bool quads(int width, const void* a, const void* b, const void* c, const void* d, const void* e, const void* f) {
    return width % 4 == 0 && !(((uintptr_t)a | (uintptr_t)b | (uintptr_t)c | (uintptr_t)d | (uintptr_t)e | (uintptr_t)f) & 15);
}

template <typename T>
int tanh_rows(const float* x, const int* rows, Tanh norm, void* out, int count, int width, cudaStream_t stream) {
    const bool four = quads(width, x, norm.weight, norm.bias, out, nullptr, nullptr);
    const size_t total = (size_t)count * width / (four ? 4 : 1);
    const dim3 grid((unsigned)((total + 255) / 256));
    if (four)
        MB_LAUNCH("tanh_rows", (tanh_rows_kernel<T, 4>), grid, dim3(256), 0, stream, true, x, rows, norm, (T*)out, total, width);
    else
        MB_LAUNCH("tanh_rows", (tanh_rows_kernel<T, 1>), grid, dim3(256), 0, stream, true, x, rows, norm, (T*)out, total, width);
    return 0;
}

template <typename T>
int tanh_add(float* x, const float* y, ExpertSum sum, Tanh norm, Then then, void* out, int count, int width, cudaStream_t stream) {
    const bool four = quads(width, x, y, norm.weight, norm.bias, out, nullptr) && quads(width, then.norm.weight, then.norm.bias, nullptr, nullptr, nullptr, nullptr);
    const size_t total = (size_t)count * width / (four ? 4 : 1);
    const dim3 grid((unsigned)((total + 255) / 256));
    if (four)
        MB_LAUNCH("tanh_add", (tanh_add_kernel<T, 4>), grid, dim3(256), 0, stream, true, x, y, sum, norm, then, (T*)out, total, width);
    else
        MB_LAUNCH("tanh_add", (tanh_add_kernel<T, 1>), grid, dim3(256), 0, stream, true, x, y, sum, norm, then, (T*)out, total, width);
    return 0;
}

template <typename T>
int rms_add(float* x, const float* y, const float* weight, float eps, Then then, void* out, int count, int width, cudaStream_t stream) {
    const bool four = quads(width, x, y, weight, out, then.norm.weight, then.norm.bias);
    const int vec = four ? 4 : 1;
    int threads = 32;
    while (threads < 1024 && threads * vec < width) threads *= 2;
    const int kept = (width + threads * vec - 1) / (threads * vec);
#define MB_RMS(VEC, KEPT)                                                                                                                 \
    if (four == (VEC == 4) && kept <= KEPT) {                                                                                             \
        MB_LAUNCH("rms_add", (rms_add_kernel<T, VEC, KEPT>), dim3(count), dim3(threads), 0, stream, true, x, y, weight, eps, then, (T*)out, width); \
        return 0;                                                                                                                         \
    }
    MB_RMS(4, 1)
    MB_RMS(4, 4)
    MB_RMS(1, 1)
    MB_RMS(1, 4)
    MB_RMS(1, 16)
#undef MB_RMS
    return fail("rms_add: rows of %d numbers exceed 16384", width);
}

}  // namespace mb

using namespace mb;

// out [count, width] (storage type) = tanh(alpha * x[row]) * weight + bias; rows: which rows of x (null: all, in order).
MB_EXPORT int mb_tanh_rows(const float* x, const int* rows, float alpha, const float* weight, const float* bias, void* out, int dtype,
                           int count, int width, cudaStream_t stream) {
    if (count <= 0 || width <= 0) return 0;
    const Tanh norm{alpha, weight, bias};
    int status;
    if (dtype == MB_F32) status = tanh_rows<float>(x, rows, norm, out, count, width, stream);
    else if (dtype == MB_BF16) status = tanh_rows<__nv_bfloat16>(x, rows, norm, out, count, width, stream);
    else return fail("tanh_rows: unknown dtype code %d", dtype);
    return status ? status : check_launch("tanh_rows");
}

// y: [count, width] (top 0), or expert results (top > 0: see ExpertSum).  then_kind 0 / 1 / 2: see Then; out may be null for 0.
MB_EXPORT int mb_result_tanh_add(float* x, const float* y, const int* position, int top, float entry_weight, float alpha,
                                 const float* weight, const float* bias, int then_kind, float then_alpha, const float* then_weight,
                                 const float* then_bias, void* out, int dtype, int count, int width, cudaStream_t stream) {
    if (count <= 0 || width <= 0) return 0;
    if (then_kind < 0 || then_kind > 2 || (then_kind != 0 && out == nullptr) || (then_kind == 2 && (then_weight == nullptr || then_bias == nullptr)))
        return fail("result_tanh_add: what follows (%d) lacks its tensors", then_kind);
    const ExpertSum sum{position, top, entry_weight};
    const Tanh norm{alpha, weight, bias};
    const Then then{then_kind, {then_alpha, then_weight, then_bias}};
    int status;
    if (dtype == MB_F32) status = tanh_add<float>(x, y, sum, norm, then, out, count, width, stream);
    else if (dtype == MB_BF16) status = tanh_add<__nv_bfloat16>(x, y, sum, norm, then, out, count, width, stream);
    else return fail("result_tanh_add: unknown dtype code %d", dtype);
    return status ? status : check_launch("result_tanh_add");
}

MB_EXPORT int mb_result_rms_add(float* x, const float* y, const float* weight, float eps, int then_kind, float then_alpha,
                                const float* then_weight, const float* then_bias, void* out, int dtype, int count, int width,
                                cudaStream_t stream) {
    if (count <= 0 || width <= 0) return 0;
    if (then_kind < 0 || then_kind > 2 || (then_kind != 0 && out == nullptr) || (then_kind == 2 && (then_weight == nullptr || then_bias == nullptr)))
        return fail("result_rms_add: what follows (%d) lacks its tensors", then_kind);
    const Then then{then_kind, {then_alpha, then_weight, then_bias}};
    int status;
    if (dtype == MB_F32) status = rms_add<float>(x, y, weight, eps, then, out, count, width, stream);
    else if (dtype == MB_BF16) status = rms_add<__nv_bfloat16>(x, y, weight, eps, then, out, count, width, stream);
    else return fail("result_rms_add: unknown dtype code %d", dtype);
    return status ? status : check_launch("result_rms_add");
}

// gate float rows (stride in elements); table [vocab, dim] and out [rows, columns] in the storage type, columns >= dim.
MB_EXPORT int mb_side_gate(const float* gate, int gate_stride, const void* table, const int* tokens, int dim, void* out, int columns,
                           int dtype, int rows, cudaStream_t stream) {
    if (rows <= 0 || columns <= 0) return 0;
    if (dim > columns) return fail("side_gate: %d numbers do not fit rows of %d", dim, columns);
    const size_t total = (size_t)rows * columns;
    const dim3 grid((unsigned)((total + 255) / 256));
    if (dtype == MB_F32)
        MB_LAUNCH("side_gate", side_gate_kernel<float>, grid, dim3(256), 0, stream, true, gate, gate_stride, (const float*)table, tokens, dim,
                  (float*)out, columns, total);
    else if (dtype == MB_BF16)
        MB_LAUNCH("side_gate", side_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, true, gate, gate_stride, (const __nv_bfloat16*)table,
                  tokens, dim, (__nv_bfloat16*)out, columns, total);
    else
        return fail("side_gate: unknown dtype code %d", dtype);
    return check_launch("side_gate");
}
