// A layer norm with weight and bias behind the sum of pending updates to the 32-bit residual stream:
//   residual += delta_a + delta_b (each null: none);
//   out = (residual - mean) / sqrt(mean((residual - mean)^2) + eps) * w + b, row by row, 32-bit.
// The deviations are summed in a second pass over the row (which lies in shared memory or registers): the difference of
// two large sums would lose the variance of a row whose mean is far from zero.
#include "common.cuh"

namespace {

// A CTA a row, the row in shared memory.
template <typename T>
__global__ void __launch_bounds__(512)
add_layer_norm_kernel(float* __restrict__ res, const T* __restrict__ delta_a, const T* __restrict__ delta_b,
                      const float* __restrict__ w, const float* __restrict__ b, float eps, T* __restrict__ out, int d, int vec) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * d;
    constexpr int N = Vec16<T>::N;
    const bool any = delta_a != nullptr || delta_b != nullptr;
    float sum = 0.f;
    if (vec) {
        for (int i = threadIdx.x * N; i < d; i += blockDim.x * N) {
            float v[N], dv[N];
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 x = *reinterpret_cast<const float4*>(res + base + i + j);
                v[j] = x.x; v[j + 1] = x.y; v[j + 2] = x.z; v[j + 3] = x.w;
            }
            if (delta_a != nullptr) {
                Vec16<T>::load(delta_a + base + i, dv);
#pragma unroll
                for (int j = 0; j < N; ++j) v[j] += dv[j];
            }
            if (delta_b != nullptr) {
                Vec16<T>::load(delta_b + base + i, dv);
#pragma unroll
                for (int j = 0; j < N; ++j) v[j] += dv[j];
            }
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 x = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
                if (any) *reinterpret_cast<float4*>(res + base + i + j) = x;
                *reinterpret_cast<float4*>(row + i + j) = x;
                sum += (x.x + x.y) + (x.z + x.w);
            }
        }
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            float v = res[base + i];
            if (delta_a != nullptr) v += to_f32(delta_a[base + i]);
            if (delta_b != nullptr) v += to_f32(delta_b[base + i]);
            if (any) res[base + i] = v;
            row[i] = v;
            sum += v;
        }
    }
    const float mean = block_sum(sum, red) / (float)d;
    float sq = 0.f;
    if (vec) {                                             // every thread its own elements again
        for (int i = threadIdx.x * N; i < d; i += blockDim.x * N) {
#pragma unroll
            for (int j = 0; j < N; ++j) { const float c = row[i + j] - mean; sq = fmaf(c, c, sq); }
        }
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) { const float c = row[i] - mean; sq = fmaf(c, c, sq); }
    }
    const float inv = 1.f / sqrtf(block_sum(sq, red) / (float)d + eps);
    if (vec) {
        for (int i = threadIdx.x * N; i < d; i += blockDim.x * N) {
            float v[N];
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 wv = *reinterpret_cast<const float4*>(w + i + j), bv = *reinterpret_cast<const float4*>(b + i + j);
                v[j] = fmaf((row[i + j] - mean) * inv, wv.x, bv.x);
                v[j + 1] = fmaf((row[i + j + 1] - mean) * inv, wv.y, bv.y);
                v[j + 2] = fmaf((row[i + j + 2] - mean) * inv, wv.z, bv.z);
                v[j + 3] = fmaf((row[i + j + 3] - mean) * inv, wv.w, bv.w);
            }
            Vec16<T>::store(out + base + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) out[base + i] = from_f32<T>(fmaf((row[i] - mean) * inv, w[i], b[i]));
    }
}

// Many rows: a warp a row, the row in registers (CH 16-byte chunks of the output type a lane), no barriers.
template <typename T, int CH>
__global__ void __launch_bounds__(128)
add_layer_norm_rows_kernel(float* __restrict__ res, const T* __restrict__ delta_a, const T* __restrict__ delta_b,
                           const float* __restrict__ w, const float* __restrict__ b, float eps, T* __restrict__ out, int n,
                           int d) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int N = Vec16<T>::N;
    const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (r >= n) return;
    const size_t base = (size_t)r * d;
    const bool any = delta_a != nullptr || delta_b != nullptr;
    float v[CH][N];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = (lane + 32 * k) * N;
        if (i < d) {
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 x = *reinterpret_cast<const float4*>(res + base + i + j);
                v[k][j] = x.x; v[k][j + 1] = x.y; v[k][j + 2] = x.z; v[k][j + 3] = x.w;
            }
            float dv[N];
            if (delta_a != nullptr) {
                Vec16<T>::load(delta_a + base + i, dv);
#pragma unroll
                for (int j = 0; j < N; ++j) v[k][j] += dv[j];
            }
            if (delta_b != nullptr) {
                Vec16<T>::load(delta_b + base + i, dv);
#pragma unroll
                for (int j = 0; j < N; ++j) v[k][j] += dv[j];
            }
            if (any) {
#pragma unroll
                for (int j = 0; j < N; j += 4)
                    *reinterpret_cast<float4*>(res + base + i + j) = make_float4(v[k][j], v[k][j + 1], v[k][j + 2], v[k][j + 3]);
            }
#pragma unroll
            for (int j = 0; j < N; ++j) sum += v[k][j];
        }
    }
    const float mean = warp_sum(sum) / (float)d;
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        if ((lane + 32 * k) * N < d) {
#pragma unroll
            for (int j = 0; j < N; ++j) { const float c = v[k][j] - mean; sq = fmaf(c, c, sq); }
        }
    }
    const float inv = 1.f / sqrtf(warp_sum(sq) / (float)d + eps);
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = (lane + 32 * k) * N;
        if (i < d) {
            float o[N];
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 wv = *reinterpret_cast<const float4*>(w + i + j), bv = *reinterpret_cast<const float4*>(b + i + j);
                o[j] = fmaf((v[k][j] - mean) * inv, wv.x, bv.x);
                o[j + 1] = fmaf((v[k][j + 1] - mean) * inv, wv.y, bv.y);
                o[j + 2] = fmaf((v[k][j + 2] - mean) * inv, wv.z, bv.z);
                o[j + 3] = fmaf((v[k][j + 3] - mean) * inv, wv.w, bv.w);
            }
            Vec16<T>::store(out + base + i, o);
        }
    }
}

template <typename T, int CH>
void launch_rows(float* res, const T* da, const T* db, const float* w, const float* b, float eps, T* out, int n, int d,
                 cudaStream_t stream) {
    tis_launch(add_layer_norm_rows_kernel<T, CH>, dim3((n + 3) / 4), dim3(128), 0, stream, res, da, db, w, b, eps, out, n, d);
}

}  // namespace

TIS_API int tis_add_layer_norm(int dtype, float* residual, const void* delta_a, const void* delta_b, const float* w,
                               const float* b, float eps, void* out, int n, int d, cudaStream_t stream) {
    if (n <= 0) return TIS_OK;
    const size_t smem = (size_t)d * sizeof(float);
    if (d <= 0 || smem > 96 * 1024 || w == nullptr || b == nullptr || out == nullptr) {
        tis_set_error("add_layer_norm: width %d (one row must fit 96 KB of shared memory), or no weight, bias or output", d);
        return TIS_BAD_SIZE;
    }
    const int per_lane = dtype == TIS_BF16 ? 8 : 4;
    const int vec = d % per_lane == 0 &&
                    (((uintptr_t)residual | (uintptr_t)delta_a | (uintptr_t)delta_b | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out) % 16) == 0;
    const int chunks = (d + 32 * per_lane - 1) / (32 * per_lane);
    if (n >= 1024 && vec && chunks <= 8) {
        TIS_DISPATCH_DTYPE(dtype, T, {
            const T* da = (const T*)delta_a;
            const T* db = (const T*)delta_b;
            if (chunks <= 2) launch_rows<T, 2>(residual, da, db, w, b, eps, (T*)out, n, d, stream);
            else if (chunks <= 4) launch_rows<T, 4>(residual, da, db, w, b, eps, (T*)out, n, d, stream);
            else if (chunks <= 6) launch_rows<T, 6>(residual, da, db, w, b, eps, (T*)out, n, d, stream);
            else launch_rows<T, 8>(residual, da, db, w, b, eps, (T*)out, n, d, stream);
        });
        return tis_check_launch("add_layer_norm");
    }
    const int threads = d >= 2048 ? 512 : 256;
    TIS_DISPATCH_DTYPE(dtype, T, {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(add_layer_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        tis_launch(add_layer_norm_kernel<T>, dim3(n), dim3(threads), smem, stream, residual, (const T*)delta_a,
                   (const T*)delta_b, w, b, eps, (T*)out, d, vec);
    });
    return tis_check_launch("add_layer_norm");
}
