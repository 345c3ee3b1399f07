// Between the projections and the cache of an attention whose queries and keys are rotated by their position and then
// divided by their root mean square, head by head.  A row of `qkv` holds H query heads and G key heads of `dim` elements,
// then G value heads of `v_dim`:
//   the first `rot` elements of every query and key head are rotated by the row's position (element 2i with 2i + 1, or i with
//   i + rot / 2; cos, sin: [positions][rot / 2]); with `norm` the whole head is then divided by sqrt(mean of squares + eps);
//   queries stay where they are, keys and values go into the row's page.
// `G` 0: a row holds queries only and nothing is written into the cache (a layer that reads another layer's keys).
// Pages: element (page, kv head, position in the page, i) at pages + page * page_stride + head * head_stride +
// position * width + i; with `permuted` the 16-byte chunks of a row are permuted by the position (cache_chunk in common.cuh:
// the row format of the attention kernels whose keys and values have one width).  Everything is computed in 32-bit; T is the storage type.
#include "common.cuh"

namespace {

struct RotateNorm {
    int ld, H, G, dim, v_dim, rot, interleaved, norm, permuted;
    float eps;
    const float* cos_t;
    const float* sin_t;
    size_t k_page_stride, k_head_stride, v_page_stride, v_head_stride;
    int page_size, num_pages;
    const int* block_table; int bt_stride;
    const int* positions; const int* row_slot;
    int* fault;
    int n;
};

__device__ __forceinline__ int page_of(const RotateNorm& p, int slot, int pos, bool report) {
    const int page = p.block_table[(size_t)slot * p.bt_stride + pos / p.page_size];
    if (page < 0 || page >= p.num_pages) {
        if (report) atomicExch(p.fault, 5);
        return -1;
    }
    return page;
}

// Neighbouring elements paired, whole 16-byte vectors: LPH lanes share a head, VPL vectors each, so that a rotation pair
// lies in one lane's registers and the sum of squares is a shuffle among the lanes of the head.
template <typename T, int LPH, int VPL>
__global__ void __launch_bounds__(256)
rotate_norm_vec_kernel(T* __restrict__ qkv, T* __restrict__ k_pages, T* __restrict__ v_pages, const RotateNorm p) {
    constexpr int N = Vec16<T>::N;
    pdl_launch_dependents();
    const int per_row = p.H + 2 * p.G;
    const int item = (int)((blockIdx.x * blockDim.x + threadIdx.x) / LPH);
    const int lane = threadIdx.x % LPH;
    const int r = item / per_row, hh = item - r * per_row;
    const int slot = r < p.n ? p.row_slot[r] : -1;
    const bool live = slot >= 0;
    const int pos = live ? p.positions[r] : 0;
    const bool is_q = hh < p.H, is_v = hh >= p.H + p.G;
    int page = -1;
    if (live && !is_q) page = page_of(p, slot, pos, lane == 0);
    float cs[VPL][N / 2], sn[VPL][N / 2];
    if (live && !is_v) {                                      // the tables do not depend on the kernel before
        const float* ct = p.cos_t + (size_t)pos * (p.rot >> 1);
        const float* st = p.sin_t + (size_t)pos * (p.rot >> 1);
#pragma unroll
        for (int k = 0; k < VPL; ++k) {
            const int e = (lane + LPH * k) * N;
            if (N == 8 && (p.rot & 7) == 0) {                 // a vector is rotated as a whole or not at all
                const bool in = e < p.rot;
                const float4 c4 = in ? *reinterpret_cast<const float4*>(ct + (e >> 1)) : make_float4(1.f, 1.f, 1.f, 1.f);
                const float4 s4 = in ? *reinterpret_cast<const float4*>(st + (e >> 1)) : make_float4(0.f, 0.f, 0.f, 0.f);
                cs[k][0] = c4.x; cs[k][1] = c4.y; cs[k][N / 2 - 2] = c4.z; cs[k][N / 2 - 1] = c4.w;
                sn[k][0] = s4.x; sn[k][1] = s4.y; sn[k][N / 2 - 2] = s4.z; sn[k][N / 2 - 1] = s4.w;
                continue;
            }
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const bool in = e + 2 * j < p.rot;
                cs[k][j] = in ? ct[(e >> 1) + j] : 1.f;
                sn[k][j] = in ? st[(e >> 1) + j] : 0.f;
            }
        }
    }
    pdl_wait();
    T* row = qkv + (size_t)(live ? r : 0) * p.ld;
    const int in_page = pos % p.page_size;
    if (is_v) {                                               // (a warp may hold value heads beside others: no return)
        if (page >= 0) {
            const int g = hh - p.H - p.G;
            const T* src = row + (size_t)(p.H + p.G) * p.dim + (size_t)g * p.v_dim;
            T* dst = v_pages + (size_t)page * p.v_page_stride + (size_t)g * p.v_head_stride + (size_t)in_page * p.v_dim;
            const int nch = p.v_dim / N;
            for (int i = lane * N; i < p.v_dim; i += LPH * N)
                *reinterpret_cast<uint4*>(dst + (p.permuted ? cache_chunk(i / N, pos, nch) * N : i)) = *reinterpret_cast<const uint4*>(src + i);
        }
    }
    const bool works = live && !is_v && (is_q || page >= 0);
    T* src = row + (size_t)(is_v ? 0 : hh) * p.dim;
    float v[VPL][N];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPL; ++k) {
        const int e = (lane + LPH * k) * N;
        if (works && e < p.dim) {
            Vec16<T>::load(src + e, v[k]);
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const float a = v[k][2 * j], b = v[k][2 * j + 1];
                v[k][2 * j] = a * cs[k][j] - b * sn[k][j];
                v[k][2 * j + 1] = b * cs[k][j] + a * sn[k][j];
            }
#pragma unroll
            for (int j = 0; j < N; ++j) ss = fmaf(v[k][j], v[k][j], ss);
        }
    }
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!works) return;
    const float f = p.norm ? 1.f / sqrtf(ss / (float)p.dim + p.eps) : 1.f;
    T* dst = is_q ? src : k_pages + (size_t)page * p.k_page_stride + (size_t)(hh - p.H) * p.k_head_stride + (size_t)in_page * p.dim;
#pragma unroll
    for (int k = 0; k < VPL; ++k) {
        const int e = (lane + LPH * k) * N;
        if (e < p.dim) {
#pragma unroll
            for (int j = 0; j < N; ++j) v[k][j] *= f;
            Vec16<T>::store(dst + (p.permuted && !is_q ? cache_chunk(e / N, pos, p.dim / N) * N : e), v[k]);
        }
    }
}

// Any size and pairing: a CTA a row, a warp a head.  A lane owns whole rotation pairs, so that queries can be replaced in
// place: the first pass sums the squares, the second makes the values again and stores them.
template <typename T>
__global__ void __launch_bounds__(128)
rotate_norm_kernel(T* __restrict__ qkv, T* __restrict__ k_pages, T* __restrict__ v_pages, const RotateNorm p) {
    pdl_launch_dependents();
    const int r = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int slot = p.row_slot[r];
    if (slot < 0) return;
    const int pos = p.positions[r];
    const int half = p.rot >> 1;
    const float* ct = p.cos_t + (size_t)pos * half;
    const float* st = p.sin_t + (size_t)pos * half;
    const int page = p.G > 0 ? page_of(p, slot, pos, threadIdx.x == 0) : -1;
    const int in_page = pos % p.page_size;
    pdl_wait();
    T* row = qkv + (size_t)r * p.ld;
    constexpr int N = Vec16<T>::N;
    auto place = [&](int i, int width, bool permuted) {
        return permuted ? cache_chunk(i / N, pos, width / N) * N + i % N : i;
    };
    const int heads = p.H + (page >= 0 ? p.G : 0);
    for (int hh = warp; hh < heads; hh += nw) {
        T* src = row + (size_t)hh * p.dim;
        const bool perm = p.permuted && hh >= p.H;
        T* dst = hh < p.H ? src : k_pages + (size_t)page * p.k_page_stride + (size_t)(hh - p.H) * p.k_head_stride + (size_t)in_page * p.dim;
        float ss = 0.f;
        for (int i = lane; i < half; i += 32) {
            const int ia = p.interleaved ? 2 * i : i, ib = p.interleaved ? 2 * i + 1 : i + half;
            const float a = to_f32(src[ia]), b = to_f32(src[ib]);
            const float x = a * ct[i] - b * st[i], y = b * ct[i] + a * st[i];
            ss = fmaf(x, x, fmaf(y, y, ss));
        }
        for (int i = p.rot + lane; i < p.dim; i += 32) { const float x = to_f32(src[i]); ss = fmaf(x, x, ss); }
        ss = warp_sum(ss);
        const float f = p.norm ? 1.f / sqrtf(ss / (float)p.dim + p.eps) : 1.f;
        for (int i = lane; i < half; i += 32) {
            const int ia = p.interleaved ? 2 * i : i, ib = p.interleaved ? 2 * i + 1 : i + half;
            const float a = to_f32(src[ia]), b = to_f32(src[ib]);
            dst[place(ia, p.dim, perm)] = from_f32<T>((a * ct[i] - b * st[i]) * f);
            dst[place(ib, p.dim, perm)] = from_f32<T>((b * ct[i] + a * st[i]) * f);
        }
        for (int i = p.rot + lane; i < p.dim; i += 32) dst[place(i, p.dim, perm)] = from_f32<T>(to_f32(src[i]) * f);
    }
    if (page < 0) return;
    const T* vals = row + (size_t)(p.H + p.G) * p.dim;
    for (int idx = threadIdx.x; idx < p.G * p.v_dim; idx += blockDim.x) {
        const int g = idx / p.v_dim, e = idx - g * p.v_dim;
        v_pages[(size_t)page * p.v_page_stride + (size_t)g * p.v_head_stride + (size_t)in_page * p.v_dim + place(e, p.v_dim, p.permuted)] = vals[idx];
    }
}

// The other order: queries and keys are normed first, each over all of its heads at once and with weights `w` (H * dim for the
// queries, then G * dim for the keys), and then rotated, neighbouring elements paired.  Whole 16-byte vectors, a CTA takes
// `rows` rows one after the other, VPT vectors of a row a thread, whose weights stay in registers.  What does not come from the
// kernel before (weights, cosines and sines, block table) is loaded before the wait for it.
template <typename T, int VPT>
__global__ void __launch_bounds__(256)
norm_rotate_vec_kernel(T* __restrict__ qkv, T* __restrict__ k_pages, T* __restrict__ v_pages, const float* __restrict__ w,
                       const RotateNorm p, int rows) {
    constexpr int N = Vec16<T>::N;
    __shared__ float red[2][8];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nq = p.H * p.dim, nk = p.G * p.dim, total = nq + nk;
    float wv[VPT][N];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int e = (tid + k * 256) * N;
        if (e < total) {
#pragma unroll
            for (int j = 0; j < N; j += 4) {
                const float4 x = *reinterpret_cast<const float4*>(w + e + j);
                wv[k][j] = x.x; wv[k][j + 1] = x.y; wv[k][j + 2] = x.z; wv[k][j + 3] = x.w;
            }
        }
    }
    bool waited = false;
    const int r_end = min(p.n, (int)(blockIdx.x + 1) * rows);
    for (int r = blockIdx.x * rows; r < r_end; ++r) {
        const int slot = p.row_slot[r];
        if (slot < 0) continue;                               // (the same for all threads)
        const int pos = p.positions[r];
        const int page = p.G > 0 ? page_of(p, slot, pos, tid == 0) : -1;
        const int in_page = pos % p.page_size;
        const float* ct = p.cos_t + (size_t)pos * (p.rot >> 1);
        const float* st = p.sin_t + (size_t)pos * (p.rot >> 1);
        float cs[VPT][N / 2], sn[VPT][N / 2];
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int i = ((tid + k * 256) * N) % p.dim;
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const bool turns = (tid + k * 256) * N < total && i + 2 * j < p.rot;
                cs[k][j] = turns ? ct[(i >> 1) + j] : 1.f;
                sn[k][j] = turns ? st[(i >> 1) + j] : 0.f;
            }
        }
        if (!waited) { pdl_wait(); waited = true; }
        T* row = qkv + (size_t)r * p.ld;
        float v[VPT][N];
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int e = (tid + k * 256) * N;
            if (e < total) {
                Vec16<T>::load(row + e, v[k]);
                float s = 0.f;
#pragma unroll
                for (int j = 0; j < N; ++j) s = fmaf(v[k][j], v[k][j], s);
                if (e < nq) sq += s; else sk += s;
            }
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        __syncthreads();                                      // the sums of the row before have been read
        if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) { sq += red[0][i]; sk += red[1][i]; }
        const float fq = 1.f / sqrtf(sq / (float)nq + p.eps);
        const float fk = nk > 0 ? 1.f / sqrtf(sk / (float)nk + p.eps) : 0.f;
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int e = (tid + k * 256) * N;
            if (e >= total || (e >= nq && page < 0)) continue;
            const float f = e < nq ? fq : fk;
            const int hh = e / p.dim, i = e - hh * p.dim;
#pragma unroll
            for (int j = 0; j < N; ++j) v[k][j] *= f * wv[k][j];
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const float a = v[k][2 * j], b = v[k][2 * j + 1];
                v[k][2 * j] = a * cs[k][j] - b * sn[k][j];
                v[k][2 * j + 1] = b * cs[k][j] + a * sn[k][j];
            }
            if (e < nq) Vec16<T>::store(row + e, v[k]);
            else
                Vec16<T>::store(k_pages + (size_t)page * p.k_page_stride + (size_t)(hh - p.H) * p.k_head_stride + (size_t)in_page * p.dim +
                                (p.permuted ? cache_chunk(i / N, pos, p.dim / N) * N : i), v[k]);
        }
        if (page < 0) continue;
        const T* vals = row + total;
        const int nch = p.v_dim / N;
        for (int idx = tid; idx < p.G * nch; idx += 256) {
            const int g = idx / nch, c = idx - g * nch;
            *reinterpret_cast<uint4*>(v_pages + (size_t)page * p.v_page_stride + (size_t)g * p.v_head_stride + (size_t)in_page * p.v_dim +
                                      (p.permuted ? cache_chunk(c, pos, nch) : c) * N) = *reinterpret_cast<const uint4*>(vals + idx * N);
        }
    }
}

// The same for any size and pairing.  A thread owns whole rotation pairs, so that queries can be replaced in place.
template <typename T>
__global__ void __launch_bounds__(256)
norm_rotate_kernel(T* __restrict__ qkv, T* __restrict__ k_pages, T* __restrict__ v_pages, const float* __restrict__ w,
                   const RotateNorm p) {
    __shared__ float red[33];
    pdl_launch_dependents();
    const int r = blockIdx.x, tid = threadIdx.x;
    const int slot = p.row_slot[r];
    if (slot < 0) return;
    const int pos = p.positions[r];
    const int page = p.G > 0 ? page_of(p, slot, pos, tid == 0) : -1;
    const int in_page = pos % p.page_size;
    const int half = p.rot >> 1;
    const float* ct = p.cos_t + (size_t)pos * half;
    const float* st = p.sin_t + (size_t)pos * half;
    const int nq = p.H * p.dim, nk = p.G * p.dim;
    pdl_wait();
    T* row = qkv + (size_t)r * p.ld;
    constexpr int N = Vec16<T>::N;
    auto place = [&](int i, int width, bool permuted) {
        return permuted ? cache_chunk(i / N, pos, width / N) * N + i % N : i;
    };
    float sq = 0.f, sk = 0.f;
    for (int e = tid; e < nq + nk; e += blockDim.x) {
        const float x = to_f32(row[e]);
        if (e < nq) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
    }
    const float fq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + p.eps);
    const float fk = nk > 0 ? 1.f / sqrtf(block_sum(sk, red) / (float)nk + p.eps) : 0.f;
    const int heads = p.H + (page >= 0 ? p.G : 0);
    const int units = half + (p.dim - p.rot);                 // rotation pairs and single elements of a head
    for (int idx = tid; idx < heads * units; idx += blockDim.x) {
        const int hh = idx / units, u = idx - hh * units;
        T* src = row + (size_t)hh * p.dim;
        const float* wh = w + (size_t)hh * p.dim;
        const bool perm = p.permuted && hh >= p.H;
        const float f = hh < p.H ? fq : fk;
        T* dst = hh < p.H ? src : k_pages + (size_t)page * p.k_page_stride + (size_t)(hh - p.H) * p.k_head_stride + (size_t)in_page * p.dim;
        if (u < half) {
            const int ia = p.interleaved ? 2 * u : u, ib = p.interleaved ? 2 * u + 1 : u + half;
            const float a = to_f32(src[ia]) * f * wh[ia], b = to_f32(src[ib]) * f * wh[ib];
            dst[place(ia, p.dim, perm)] = from_f32<T>(a * ct[u] - b * st[u]);
            dst[place(ib, p.dim, perm)] = from_f32<T>(b * ct[u] + a * st[u]);
        } else {
            const int i = p.rot + u - half;
            dst[place(i, p.dim, perm)] = from_f32<T>(to_f32(src[i]) * f * wh[i]);
        }
    }
    if (page < 0) return;
    const T* vals = row + nq + nk;
    for (int idx = tid; idx < p.G * p.v_dim; idx += blockDim.x) {
        const int g = idx / p.v_dim, e = idx - g * p.v_dim;
        v_pages[(size_t)page * p.v_page_stride + (size_t)g * p.v_head_stride + (size_t)in_page * p.v_dim + place(e, p.v_dim, p.permuted)] = vals[idx];
    }
}

template <typename T>
void launch_norm_rotate(T* qkv, T* k_pages, T* v_pages, const float* w, const RotateNorm& p, bool vec, cudaStream_t stream) {
    const int per = ((p.H + p.G) * p.dim / Vec16<T>::N + 255) / 256;
    // rows a CTA takes: enough CTAs for four on every SM, a thread's weights loaded once for all of its rows
    const int rows = p.n >= 2 * 4 * 148 ? (p.n / (4 * 148) < 8 ? p.n / (4 * 148) : 8) : 1;
    const dim3 grid((p.n + rows - 1) / rows);
    if (!vec || per > 8 || (uintptr_t)w % 16) tis_launch(norm_rotate_kernel<T>, dim3(p.n), dim3(256), 0, stream, qkv, k_pages, v_pages, w, p);
    else if (per <= 1) tis_launch(norm_rotate_vec_kernel<T, 1>, grid, dim3(256), 0, stream, qkv, k_pages, v_pages, w, p, rows);
    else if (per <= 2) tis_launch(norm_rotate_vec_kernel<T, 2>, grid, dim3(256), 0, stream, qkv, k_pages, v_pages, w, p, rows);
    else if (per <= 4) tis_launch(norm_rotate_vec_kernel<T, 4>, grid, dim3(256), 0, stream, qkv, k_pages, v_pages, w, p, rows);
    else tis_launch(norm_rotate_vec_kernel<T, 8>, grid, dim3(256), 0, stream, qkv, k_pages, v_pages, w, p, rows);
}

template <typename T, int LPH, int VPL>
void launch_vec(T* qkv, T* k_pages, T* v_pages, const RotateNorm& p, cudaStream_t stream) {
    const size_t threads = (size_t)p.n * (p.H + 2 * p.G) * LPH;
    tis_launch(rotate_norm_vec_kernel<T, LPH, VPL>, dim3((unsigned)((threads + 255) / 256)), dim3(256), 0, stream, qkv, k_pages,
               v_pages, p);
}

template <typename T>
void launch_any(T* qkv, T* k_pages, T* v_pages, const RotateNorm& p, bool vec, cudaStream_t stream) {
    const int nv = p.dim / Vec16<T>::N;
    if (!vec || nv > 128) {
        tis_launch(rotate_norm_kernel<T>, dim3(p.n), dim3(128), 0, stream, qkv, k_pages, v_pages, p);
    } else if (nv <= 4) launch_vec<T, 4, 1>(qkv, k_pages, v_pages, p, stream);
    else if (nv <= 8) launch_vec<T, 8, 1>(qkv, k_pages, v_pages, p, stream);
    else if (nv <= 16) launch_vec<T, 16, 1>(qkv, k_pages, v_pages, p, stream);
    else if (nv <= 32) launch_vec<T, 32, 1>(qkv, k_pages, v_pages, p, stream);
    else if (nv <= 64) launch_vec<T, 32, 2>(qkv, k_pages, v_pages, p, stream);
    else launch_vec<T, 32, 4>(qkv, k_pages, v_pages, p, stream);
}

}  // namespace

// `whole_w` (null: none; else (H + G) * dim weights): the norm comes before the rotation and runs over all query heads, and over
// all key heads, at once (`norm` is then not looked at).
TIS_API int tis_rotate_norm_store(int dtype, void* qkv, int ld, int H, int G, int dim, int v_dim, int rot, int interleaved,
                                  int permuted, const float* cos_t, const float* sin_t, int norm, float eps,
                                  const float* whole_w, void* k_pages,
                                  size_t k_page_stride, size_t k_head_stride, void* v_pages, size_t v_page_stride,
                                  size_t v_head_stride, int page_size, int num_pages, const int* block_table, int bt_stride,
                                  const int* positions, const int* row_slot, int* fault, int n, cudaStream_t stream) {
    if (n <= 0) return TIS_OK;
    if (H <= 0 || G < 0 || dim <= 0 || (G > 0 && v_dim <= 0) || rot < 0 || rot % 2 || rot > dim || page_size <= 0 ||
        ld < H * dim + G * (dim + v_dim) || (size_t)n * (H + 2 * G) * 32 > 0x7fffffffull) {
        tis_set_error("rotate_norm_store: %d rows of %d elements, %d heads, %d kv heads of %d and %d elements, %d of them rotated",
                      n, ld, H, G, dim, v_dim, rot);
        return TIS_BAD_SIZE;
    }
    RotateNorm p;
    p.ld = ld; p.H = H; p.G = G; p.dim = dim; p.v_dim = v_dim; p.rot = rot; p.interleaved = interleaved; p.permuted = permuted; p.norm = norm; p.eps = eps;
    p.cos_t = cos_t; p.sin_t = sin_t;
    p.k_page_stride = k_page_stride; p.k_head_stride = k_head_stride; p.v_page_stride = v_page_stride; p.v_head_stride = v_head_stride;
    p.page_size = page_size; p.num_pages = num_pages; p.block_table = block_table; p.bt_stride = bt_stride;
    p.positions = positions; p.row_slot = row_slot; p.fault = fault; p.n = n;
    const size_t N = dtype == TIS_BF16 ? 8 : 4;
    if (permuted && G > 0 && (dim % N || v_dim % N)) {
        tis_set_error("rotate_norm_store: rows of %d and %d elements are not whole 16-byte chunks", dim, v_dim);
        return TIS_BAD_SIZE;
    }
    const bool vec = (interleaved || rot == 0) && dim % N == 0 && ld % N == 0 && (uintptr_t)qkv % 16 == 0 &&
                     (G == 0 || (v_dim % N == 0 && ((k_page_stride | k_head_stride | v_page_stride | v_head_stride) % N) == 0 &&
                                 ((uintptr_t)k_pages | (uintptr_t)v_pages) % 16 == 0));
    if (whole_w != nullptr) {
        TIS_DISPATCH_DTYPE(dtype, T, launch_norm_rotate<T>((T*)qkv, (T*)k_pages, (T*)v_pages, whole_w, p, vec, stream));
        return tis_check_launch("norm_rotate_store");
    }
    TIS_DISPATCH_DTYPE(dtype, T, launch_any<T>((T*)qkv, (T*)k_pages, (T*)v_pages, p, vec, stream));
    return tis_check_launch("rotate_norm_store");
}
