// Steps around the sublayers of a pre-norm decoder whose sublayers' results are scaled value by value, and a per-layer input from the token
// itself at a layer's end.
//
//  residual_step  everything that happens to a token's float32 residual row between two sublayers, one block a row:
//                   x += c . y                          what a sublayer ADDED into the zeroed row y, scaled (c null: nothing), then y = 0
//                   x += m (z / sqrt(mean(z^2) + eps)) . wz      (z null: nothing)
//                   x += E[id]  (E null: nothing);   x += v  (v null: nothing)
//                   out = LN(x; wn, bn), or x itself, in the compute dtype  (out null: nothing)
//  token_gate     g = gelu(a) . S[id, off .. off + dim], gelu in its tanh form, a float32 [T, dim]
//  token_side     for few tokens, residual_step with the per-layer input worked out in it: a = G (x + c . y), g = gelu(a) . S[id, ..], z = P g.
//                   A cluster of eight blocks takes a token.  Each works out its share of a's rows and leaves their g in every block's shared
//                   memory, then its share of z's rows; the sum of z's squares and the parts of the layer norm (mean and squared deviations
//                   of each block's own columns, put together exactly) meet through distributed shared memory.
//
// A row's sums meet in an order that depends on the width alone.  All arithmetic is float32 with accurate tanhf, division and sqrtf.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace vk {

constexpr int RS_KEEP = 4;      // 16-byte pieces of a row that a thread keeps

template <typename T> __device__ __forceinline__ void rs_store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void rs_store4<float>(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void rs_store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

template <typename T> __device__ __forceinline__ float4 rs_load4(const T* p);
template <> __device__ __forceinline__ float4 rs_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 rs_load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}

template <typename T>
struct StepArgs {
    float* x;                   // [rows][n]
    float* y;                   // [rows][n] or null
    const float* c;             // [n] or null
    const float* z;             // [rows][n] or null
    const float* wz;            // [n]
    const T* table;             // [vocab][n] or null
    const int32_t* ids;         // [rows]
    const float* add;           // [n] or null
    const float* wn;            // [n] or null: a layer norm with bn
    const float* bn;
    T* out;                     // [rows][n] or null
    int n, vocab;
    float eps, mult;
};

__device__ __forceinline__ int rs_id(const int32_t* ids, int t, int vocab) {
    const int id = ids[t];
    return id < 0 || id >= vocab ? 0 : id;          // the host has checked the range; never read outside the table
}

// VEC: n a multiple of four, up to 4 * blockDim.x * RS_KEEP values, every pointer on 16 bytes (out and the table: four values): a thread's pieces
// of x, y and z are all asked for before any is used, and the row stays in registers.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) residual_step_kernel(const StepArgs<T> a) {
    __shared__ float scratch[32];
    dependency_wait();
    let_dependents_start();
    const int t = blockIdx.x, tid = threadIdx.x, n = a.n, nt = blockDim.x;
    const size_t base = (size_t)t * n;
    const T* row = a.table ? a.table + (size_t)rs_id(a.ids, t, a.vocab) * n : nullptr;
    const bool changes = a.c || a.z || row || a.add;
    if (VEC) {
        float4 u[RS_KEEP], z[RS_KEEP];
        const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int j = 0; j < RS_KEEP; j++) {
            const int i = (tid + j * nt) * 4;
            u[j] = i < n ? *reinterpret_cast<const float4*>(a.x + base + i) : zero;
            z[j] = a.z && i < n ? *reinterpret_cast<const float4*>(a.z + base + i) : zero;
            if (a.c && i < n) {
                const float4 y4 = *reinterpret_cast<const float4*>(a.y + base + i), c4 = *reinterpret_cast<const float4*>(a.c + i);
                u[j].x = fmaf(c4.x, y4.x, u[j].x); u[j].y = fmaf(c4.y, y4.y, u[j].y); u[j].z = fmaf(c4.z, y4.z, u[j].z); u[j].w = fmaf(c4.w, y4.w, u[j].w);
            }
        }
        if (a.z) {
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < RS_KEEP; j++) { ss = fmaf(z[j].x, z[j].x, ss); ss = fmaf(z[j].y, z[j].y, ss); ss = fmaf(z[j].z, z[j].z, ss); ss = fmaf(z[j].w, z[j].w, ss); }
            const float inv = a.mult / sqrtf(block_sum(ss, scratch) / (float)n + a.eps);
#pragma unroll
            for (int j = 0; j < RS_KEEP; j++) {
                const int i = (tid + j * nt) * 4;
                if (i < n) {
                    const float4 w4 = *reinterpret_cast<const float4*>(a.wz + i);
                    u[j].x = fmaf(z[j].x * inv, w4.x, u[j].x); u[j].y = fmaf(z[j].y * inv, w4.y, u[j].y);
                    u[j].z = fmaf(z[j].z * inv, w4.z, u[j].z); u[j].w = fmaf(z[j].w * inv, w4.w, u[j].w);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < RS_KEEP; j++) {
            const int i = (tid + j * nt) * 4;
            if (i >= n) continue;
            if (row) { const float4 e = rs_load4<T>(row + i); u[j].x += e.x; u[j].y += e.y; u[j].z += e.z; u[j].w += e.w; }
            if (a.add) { const float4 e = *reinterpret_cast<const float4*>(a.add + i); u[j].x += e.x; u[j].y += e.y; u[j].z += e.z; u[j].w += e.w; }
            if (changes) *reinterpret_cast<float4*>(a.x + base + i) = u[j];
            if (a.y) *reinterpret_cast<float4*>(a.y + base + i) = zero;
        }
        if (!a.out) return;
        if (!a.wn) {
#pragma unroll
            for (int j = 0; j < RS_KEEP; j++) {
                const int i = (tid + j * nt) * 4;
                if (i < n) rs_store4<T>(a.out + base + i, u[j].x, u[j].y, u[j].z, u[j].w);
            }
            return;
        }
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < RS_KEEP; j++) sum += (u[j].x + u[j].y) + (u[j].z + u[j].w);
        const float mean = block_sum(sum, scratch) / (float)n;
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < RS_KEEP; j++)
            if ((tid + j * nt) * 4 < n) {
                const float d0 = u[j].x - mean, d1 = u[j].y - mean, d2 = u[j].z - mean, d3 = u[j].w - mean;
                ss = fmaf(d0, d0, ss); ss = fmaf(d1, d1, ss); ss = fmaf(d2, d2, ss); ss = fmaf(d3, d3, ss);
            }
        const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + a.eps);
#pragma unroll
        for (int j = 0; j < RS_KEEP; j++) {
            const int i = (tid + j * nt) * 4;
            if (i < n) {
                const float4 w4 = *reinterpret_cast<const float4*>(a.wn + i), b4 = *reinterpret_cast<const float4*>(a.bn + i);
                rs_store4<T>(a.out + base + i, fmaf((u[j].x - mean) * inv, w4.x, b4.x), fmaf((u[j].y - mean) * inv, w4.y, b4.y),
                             fmaf((u[j].z - mean) * inv, w4.z, b4.z), fmaf((u[j].w - mean) * inv, w4.w, b4.w));
            }
        }
        return;
    }
    float inv_z = 0.0f;
    if (a.z) {
        float ss = 0.0f;
        for (int i = tid; i < n; i += nt) { const float v = a.z[base + i]; ss = fmaf(v, v, ss); }
        inv_z = a.mult / sqrtf(block_sum(ss, scratch) / (float)n + a.eps);
    }
    float sum = 0.0f;
    for (int i = tid; i < n; i += nt) {
        float v = a.x[base + i];
        if (a.c) v = fmaf(a.c[i], a.y[base + i], v);
        if (a.z) v = fmaf(a.z[base + i] * inv_z, a.wz[i], v);
        if (row) v += to_f32<T>(row[i]);
        if (a.add) v += a.add[i];
        if (changes) a.x[base + i] = v;
        if (a.y) a.y[base + i] = 0.0f;
        if (a.out && !a.wn) a.out[base + i] = from_f32<T>(v);
        sum += v;
    }
    if (!a.out || !a.wn) return;
    const float mean = block_sum(sum, scratch) / (float)n;
    float ss = 0.0f;
    for (int i = tid; i < n; i += nt) { const float d = a.x[base + i] - mean; ss = fmaf(d, d, ss); }       // a thread reads what it wrote itself
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + a.eps);
    for (int i = tid; i < n; i += nt) a.out[base + i] = from_f32<T>(fmaf((a.x[base + i] - mean) * inv, a.wn[i], a.bn[i]));
}

__device__ __forceinline__ float rs_gelu(float z) { return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z))); }

template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(const float* __restrict__ a, const T* __restrict__ table, int ld, int off,
                                                         const int32_t* __restrict__ ids, int vocab, T* __restrict__ out, int tokens, int dim) {
    dependency_wait();
    let_dependents_start();
    const size_t n = (size_t)tokens * dim;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(i / dim), d = (int)(i - (size_t)t * dim);
        out[i] = from_f32<T>(rs_gelu(a[i]) * to_f32<T>(table[(size_t)rs_id(ids, t, vocab) * ld + off + d]));
    }
}

constexpr int TS_BLOCKS = 8, TS_THREADS = 512, TS_WARPS = TS_THREADS / 32;

// Dot product of a row of T with float32 values in shared memory, the whole warp on one row.
template <typename T>
__device__ __forceinline__ float ts_dot(const T* __restrict__ w, const float* s, int n, int lane) {
    float acc = 0.0f;
    for (int i = lane; i < n; i += 32) acc = fmaf(s[i], to_f32<T>(w[i]), acc);
    return warp_sum(acc);
}

constexpr int TS_ROWS = 2;      // rows of the first product that a warp reads side by side
constexpr int TS_AHEAD = 8;     // pieces of the second product's rows on their way together

template <typename T>
struct SideArgs {
    const T* gate;              // G [dim][n]
    const T* proj;              // P [n][dim]
    const T* side;              // S [vocab][ld], this layer's part at off
    int ld, off, dim;
};

template <typename T>
__global__ void __launch_bounds__(TS_THREADS) token_side_kernel(const StepArgs<T> a, const SideArgs<T> sd, int vec_gate, int vec_proj) {
    extern __shared__ __align__(16) float ts_sm[];          // x + c . y [n rounded up to 4] | g [dim rounded up to 4] | z's own rows [per]
    __shared__ float scratch[32];
    __shared__ float part[2 * TS_BLOCKS], moment[2 * TS_BLOCKS];     // sums of squares, (mean, squared deviations), by block of the cluster
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), t = blockIdx.x / TS_BLOCKS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int n = a.n, dim = sd.dim, n4 = (n + 3) & ~3, d4 = (dim + 3) & ~3;
    const int per = ((n + TS_BLOCKS - 1) / TS_BLOCKS + 3) & ~3;      // columns a block
    const int lo = min(rank * per, n), hi = min(lo + per, n);
    float* xs = ts_sm;
    float* g = xs + n4;
    float* zs = g + d4;
    // the weights do not depend on the kernel before this one: on their way into the second-level cache before the wait
    {
        const char* w = reinterpret_cast<const char*>(sd.proj + (size_t)lo * dim);
        const size_t bytes = (size_t)(hi - lo) * dim * sizeof(T);
        for (size_t i = (size_t)tid * 128; i < bytes; i += (size_t)TS_THREADS * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + i));
        for (int r = rank; r < dim; r += TS_BLOCKS) {
            const char* row = reinterpret_cast<const char*>(sd.gate + (size_t)r * n);
            for (size_t i = (size_t)tid * 128; i < (size_t)n * sizeof(T); i += (size_t)TS_THREADS * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(row + i));
        }
    }
    cluster.sync();                                     // all eight blocks run: their shared memory may be written
    dependency_wait();
    let_dependents_start();
    const size_t base = (size_t)t * n;
    const int id = rs_id(a.ids, t, a.vocab);
    if (n % 4 == 0 && n4 == n && ((uintptr_t)a.x % 16) == 0 && ((uintptr_t)a.y % 16) == 0 && ((uintptr_t)a.c % 16) == 0) {
#pragma unroll 2
        for (int i = tid * 4; i < n; i += TS_THREADS * 4) {
            float4 v = *reinterpret_cast<const float4*>(a.x + base + i);
            if (a.c) {
                const float4 y4 = *reinterpret_cast<const float4*>(a.y + base + i), c4 = *reinterpret_cast<const float4*>(a.c + i);
                v.x = fmaf(c4.x, y4.x, v.x); v.y = fmaf(c4.y, y4.y, v.y); v.z = fmaf(c4.z, y4.z, v.z); v.w = fmaf(c4.w, y4.w, v.w);
            }
            *reinterpret_cast<float4*>(xs + i) = v;
        }
    } else {
        for (int i = tid; i < n; i += TS_THREADS) {
            float v = a.x[base + i];
            if (a.c) v = fmaf(a.c[i], a.y[base + i], v);
            xs[i] = v;
        }
    }
    __syncthreads();
    // a's rows, dealt out to the blocks in turn; every block gets every g
    constexpr int V = Vec16<T>::N, STRIDE = TS_WARPS * TS_BLOCKS;
    auto give = [&](int r, float s) {
        const float v = rs_gelu(s) * to_f32<T>(sd.side[(size_t)id * sd.ld + sd.off + r]);
        if (lane < TS_BLOCKS) cluster.map_shared_rank(g, lane)[r] = v;
    };
    if (vec_gate) {
        for (int r = warp * TS_BLOCKS + rank; r < dim; r += STRIDE * TS_ROWS) {
            const T* w[TS_ROWS];
            float acc[TS_ROWS];
#pragma unroll
            for (int q = 0; q < TS_ROWS; q++) { w[q] = sd.gate + (size_t)min(r + q * STRIDE, dim - 1) * n; acc[q] = 0.0f; }
#pragma unroll 4
            for (int i = lane * V; i < n; i += 32 * V) {
                float f[TS_ROWS][V];
#pragma unroll
                for (int q = 0; q < TS_ROWS; q++) load16<T>(w[q] + i, f[q]);
#pragma unroll
                for (int e = 0; e < V; e += 4) {
                    const float4 x4 = *reinterpret_cast<const float4*>(xs + i + e);
#pragma unroll
                    for (int q = 0; q < TS_ROWS; q++) {
                        acc[q] = fmaf(x4.x, f[q][e], acc[q]); acc[q] = fmaf(x4.y, f[q][e + 1], acc[q]);
                        acc[q] = fmaf(x4.z, f[q][e + 2], acc[q]); acc[q] = fmaf(x4.w, f[q][e + 3], acc[q]);
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < TS_ROWS; q++) {
                const float s = warp_sum(acc[q]);
                if (r + q * STRIDE < dim) give(r + q * STRIDE, s);
            }
        }
    } else {
        for (int r = warp * TS_BLOCKS + rank; r < dim; r += STRIDE) give(r, ts_dot<T>(sd.gate + (size_t)r * n, xs, n, lane));
    }
    // this block's rows of z; a row is dim / V pieces: several rows a warp where it is short.  The first pieces are asked for before the
    // blocks meet.
    int lanes = 1;
    while (lanes < 32 && lanes * V < dim) lanes *= 2;
    const int rows = 32 / lanes, sub = lane / lanes, in = lane - sub * lanes, step = TS_WARPS * rows, first = lo + warp * rows + sub;
    uint4 piece[TS_AHEAD];
    auto ask = [&](int r0, int i) {
#pragma unroll
        for (int q = 0; q < TS_AHEAD; q++) piece[q] = *reinterpret_cast<const uint4*>(sd.proj + (size_t)min(r0 + q * step, hi - 1) * dim + i);
    };
    if (vec_proj && first - sub < hi && in * V < dim) ask(first, in * V);
    cluster.sync();
    float ss = 0.0f;
    if (vec_proj) {
        for (int r0 = first; r0 - sub < hi; r0 += step * TS_AHEAD) {
            float acc[TS_AHEAD];
#pragma unroll
            for (int q = 0; q < TS_AHEAD; q++) acc[q] = 0.0f;
            for (int i = in * V; i < dim; i += lanes * V) {
                if (r0 != first || i != in * V) ask(r0, i);
                float gv[V];
#pragma unroll
                for (int e = 0; e < V; e += 4) *reinterpret_cast<float4*>(gv + e) = *reinterpret_cast<const float4*>(g + i + e);
#pragma unroll
                for (int q = 0; q < TS_AHEAD; q++) {
                    float f[V];
                    load16<T>(reinterpret_cast<const T*>(&piece[q]), f);
#pragma unroll
                    for (int e = 0; e < V; e++) acc[q] = fmaf(gv[e], f[e], acc[q]);
                }
            }
#pragma unroll
            for (int q = 0; q < TS_AHEAD; q++) {
                for (int o = lanes / 2; o > 0; o >>= 1) acc[q] += __shfl_xor_sync(0xffffffffu, acc[q], o);
                const int r = r0 + q * step;
                if (r < hi && in == 0) zs[r - lo] = acc[q];
            }
        }
    } else {
        for (int r = lo + warp; r < hi; r += TS_WARPS) {
            const float v = ts_dot<T>(sd.proj + (size_t)r * dim, g, dim, lane);
            if (lane == 0) zs[r - lo] = v;
        }
    }
    __syncthreads();
    for (int i = tid; i < hi - lo; i += TS_THREADS) ss = fmaf(zs[i], zs[i], ss);
    ss = block_sum(ss, scratch);
    if (tid < TS_BLOCKS) cluster.map_shared_rank(part, tid)[rank] = ss;
    cluster.sync();
    float all = 0.0f;
#pragma unroll
    for (int b = 0; b < TS_BLOCKS; b++) all += part[b];
    const float inv = a.mult / sqrtf(all / (float)n + a.eps);
    // the new row, this block's columns
    const T* row = a.table ? a.table + (size_t)id * n : nullptr;
    float sum = 0.0f;
    for (int i = lo + tid; i < hi; i += TS_THREADS) {
        float v = fmaf(zs[i - lo] * inv, a.wz[i], xs[i]);
        if (row) v += to_f32<T>(row[i]);
        if (a.add) v += a.add[i];
        a.x[base + i] = v;                              // every block has read the whole row: two barriers of the cluster ago
        if (a.y) a.y[base + i] = 0.0f;
        if (a.out && !a.wn) a.out[base + i] = from_f32<T>(v);
        xs[i] = v;
        sum += v;
    }
    if (!a.out || !a.wn) return;
    const int mine = hi - lo;
    const float own_mean = mine > 0 ? block_sum(sum, scratch) / (float)mine : 0.0f;     // the same branch for the whole block
    float dev = 0.0f;
    for (int i = lo + tid; i < hi; i += TS_THREADS) { const float d = xs[i] - own_mean; dev = fmaf(d, d, dev); }
    dev = block_sum(dev, scratch);
    if (tid < TS_BLOCKS) {
        float* m = cluster.map_shared_rank(moment, tid);
        m[2 * rank] = own_mean;
        m[2 * rank + 1] = dev;
    }
    cluster.sync();
    float mean = 0.0f;
#pragma unroll
    for (int b = 0; b < TS_BLOCKS; b++) mean += moment[2 * b] * (float)(min((b + 1) * per, n) - min(b * per, n));
    mean /= (float)n;
    float var = 0.0f;
#pragma unroll
    for (int b = 0; b < TS_BLOCKS; b++) {
        const float d = moment[2 * b] - mean;
        var += fmaf(d * d, (float)(min((b + 1) * per, n) - min(b * per, n)), moment[2 * b + 1]);
    }
    const float invn = 1.0f / sqrtf(var / (float)n + a.eps);
    for (int i = lo + tid; i < hi; i += TS_THREADS) a.out[base + i] = from_f32<T>(fmaf((xs[i] - mean) * invn, a.wn[i], a.bn[i]));
}

template <typename T>
static int launch_side(const StepArgs<T>& a, const SideArgs<T>& s, int rows, size_t smem, cudaStream_t stream) {
    constexpr int V = Vec16<T>::N;
    const int vec_gate = a.n % V == 0 && ((uintptr_t)s.gate % 16) == 0, vec_proj = s.dim % V == 0 && ((uintptr_t)s.proj % 16) == 0;
    auto kern = token_side_kernel<T>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(rows * TS_BLOCKS);
    cfg.blockDim = dim3(TS_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = TS_BLOCKS;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelEx(&cfg, kern, a, s, vec_gate, vec_proj);
}

template <typename T>
static StepArgs<T> step_args(float* x, float* y, const float* c, const float* z, const float* wz, const void* table, const int32_t* ids, int vocab,
                             const float* add, const float* wn, const float* bn, void* out, int n, float eps, float mult) {
    StepArgs<T> a;
    a.x = x; a.y = y; a.c = c; a.z = z; a.wz = wz; a.table = (const T*)table; a.ids = ids; a.add = add; a.wn = wn; a.bn = bn; a.out = (T*)out;
    a.n = n; a.vocab = vocab; a.eps = eps; a.mult = mult;
    return a;
}

}  // namespace vk

using namespace vk;

// x, y, z float32 [rows][n]; c, wz, add, wn, bn float32 [n]; table [vocab][n] and out [rows][n] in dtype; ids int32 [rows].  What is null is not
// there (see above); c needs y, z needs wz, the table needs ids, wn needs bn and out.
VK_API int vk_residual_step(float* x, float* y, const float* c, const float* z, const float* wz, const void* table, const int32_t* ids, int vocab,
                            const float* add, const float* wn, const float* bn, void* out, int rows, int n, float eps, float mult, int dtype,
                            cudaStream_t stream) {
    if (rows <= 0) return VK_OK;
    if (n <= 0 || (c && !y) || (z && !wz) || (table && (!ids || vocab <= 0)) || (wn && (!bn || !out))) return VK_BAD_SHAPE;
    auto on16 = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const int threads = n > 4 * 128 * RS_KEEP ? 256 : 128;
    const uintptr_t four = dtype == 0 ? 16 : 8;
    const bool vec = n % 4 == 0 && n <= 4 * threads * RS_KEEP && on16(x) && on16(y) && on16(c) && on16(z) && on16(wz) && on16(add) && on16(wn) && on16(bn) &&
                     ((uintptr_t)out % four) == 0 && ((uintptr_t)table % four) == 0;
    auto go = [&](auto tag) {
        using T = decltype(tag);
        const StepArgs<T> a = step_args<T>(x, y, c, z, wz, table, ids, vocab, add, wn, bn, out, n, eps, mult);
        if (vec) return launch_dependent(residual_step_kernel<T, true>, dim3(rows), dim3(threads), 0, stream, a);
        return launch_dependent(residual_step_kernel<T, false>, dim3(rows), dim3(threads), 0, stream, a);
    };
    return dtype == 0 ? go(float()) : go(__nv_bfloat16());
}

// a float32 [tokens][dim]; table [vocab][ld] in dtype, columns off .. off + dim; out [tokens][dim] in dtype.
VK_API int vk_token_gate(const float* a, const void* table, int ld, int off, const int32_t* ids, int vocab, void* out, int tokens, int dim, int dtype,
                         cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (dim <= 0 || off < 0 || off + dim > ld || vocab <= 0 || !ids) return VK_BAD_SHAPE;
    const size_t n = (size_t)tokens * dim, g = (n + 255) / 256;
    const dim3 grid((unsigned)(g > 148 * 8 ? 148 * 8 : g));
    if (dtype == 0) return launch_dependent(token_gate_kernel<float>, grid, dim3(256), 0, stream, a, (const float*)table, ld, off, ids, vocab, (float*)out, tokens, dim);
    return launch_dependent(token_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, a, (const __nv_bfloat16*)table, ld, off, ids, vocab,
                            (__nv_bfloat16*)out, tokens, dim);
}

VK_API size_t vk_token_side_smem(int n, int dim) {
    const int per = ((n + TS_BLOCKS - 1) / TS_BLOCKS + 3) & ~3;
    return (size_t)(((n + 3) & ~3) + ((dim + 3) & ~3) + per) * sizeof(float);
}

// residual_step with z = P g, g = gelu(G (x + c . y)) . side[id, off ..]: gate [dim][n], proj [n][dim], side [vocab][side_ld] in dtype; the table, if
// there is one, has as many rows as side.
VK_API int vk_token_side(float* x, float* y, const float* c, const void* gate, const void* proj, int dim, const void* side, int side_ld, int side_off,
                         const float* wz, const void* table, const int32_t* ids, int vocab, const float* add, const float* wn, const float* bn, void* out,
                         int rows, int n, float eps, float mult, int dtype, cudaStream_t stream) {
    if (rows <= 0) return VK_OK;
    if (n <= 0 || dim <= 0 || (c && !y) || !gate || !proj || !side || !wz || !ids || vocab <= 0 || side_off < 0 || side_off + dim > side_ld ||
        (wn && (!bn || !out)))
        return VK_BAD_SHAPE;
    const size_t smem = vk_token_side_smem(n, dim);
    if (smem > 200 * 1024 || rows > 65535) return VK_TOO_LARGE;
    if (dtype == 0)
        return launch_side<float>(step_args<float>(x, y, c, nullptr, wz, table, ids, vocab, add, wn, bn, out, n, eps, mult),
                                  SideArgs<float>{(const float*)gate, (const float*)proj, (const float*)side, side_ld, side_off, dim}, rows, smem, stream);
    return launch_side<__nv_bfloat16>(step_args<__nv_bfloat16>(x, y, c, nullptr, wz, table, ids, vocab, add, wn, bn, out, n, eps, mult),
                                      SideArgs<__nv_bfloat16>{(const __nv_bfloat16*)gate, (const __nv_bfloat16*)proj, (const __nv_bfloat16*)side, side_ld,
                                                              side_off, dim}, rows, smem, stream);
}
