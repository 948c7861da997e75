// The state-space mixer (structured state-space duality): a recurrent mixer whose state is, per head, a matrix S [N][P] with ONE decay
// a head and token.
//
//  a token's projections arrive as float32 columns  z (H P) | x (H P) | B (G N) | C (G N) | dt (H)  of a row of the first product
//  x, B, C   causal convolution a channel (taps weights, the last one the current token's; zeros before the sequence's start), bias, silu
//  dt        softplus(dt + bias);   log decay = -exp(A) dt                                       one each a head
//  S_t = e^(log decay) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t                          head h reads group h / (H / G) of B and C
//  out       y silu(z), divided by its root mean square in `parts` equal parts, times w
//
//  ssd_prepare     a thread a channel and eight tokens: convolution, bias, silu to the compute dtype [tokens][H P + 2 G N]; dt and the
//                  log decays to float32 [tokens][2 H].
//  ssd_recurrence  token after token, a block per (16 columns, head, segment): a warp holds four columns, the eight lanes of a column
//                  share its rows (a thread keeps DPT of them in registers).  Tokens are staged a chunk ahead in shared memory.  The
//                  form of the exact 32-bit routing and of the sizes that the chunked form (ssd_chunked.cu) does not take.
//  ssd_decode      single tokens: convolution, gates, one step and the state's update in one launch, a block per (columns, head,
//                  segment); the state's rows are on their way before the kernel waits for the product in front of it.
//  ssd_gate        a block a token: gate, norm, weight, to columns of the output product's input; further blocks move the convolution's
//                  memory of the segments on (nothing after them in the step reads the old one).
//
// A request's state row: S float32 [H][N][P], then the last taps - 1 inputs of the convolution, float32 [taps - 1][H P + 2 G N].
// Everything is float32 with accurate expf and log1pf; only what the convolution gives is rounded to the compute dtype.
#include "delta_common.cuh"

namespace vk {

constexpr int SSD_PREP_TOKENS = 8;
constexpr int SSD_THREADS = 128;
constexpr int SSD_CHUNK = 32;

// MT - 1 >= taps - 1 inputs of earlier tokens are kept (x[j] is the input j + 1 tokens back)
template <typename T, int MT>
__global__ void __launch_bounds__(256) ssd_prepare_kernel(const float* __restrict__ proj, int N, int x_off, int dt_off, const float* __restrict__ conv_w,
                                                          const float* __restrict__ conv_b, const float* __restrict__ dt_bias,
                                                          const float* __restrict__ a_log, const int32_t* __restrict__ token_seg,
                                                          const int32_t* __restrict__ seg_starts, const int32_t* __restrict__ seg_slots,
                                                          const float* __restrict__ state, size_t state_stride, size_t conv_off, T* __restrict__ xbc,
                                                          float* __restrict__ gates, int C, int H, int taps, int tokens) {
    dependency_wait();
    let_dependents_start();
    const int t0 = blockIdx.x * SSD_PREP_TOKENS, cnt = min(SSD_PREP_TOKENS, tokens - t0);
    if (blockIdx.y == gridDim.y - 1) {                      // the step sizes and the decays' logarithms
        for (int i = threadIdx.x; i < cnt * H; i += blockDim.x) {
            const int t = t0 + i / H, h = i % H;
            const float dt = softplus_f(proj[(size_t)t * N + dt_off + h] + dt_bias[h]);
            gates[(size_t)t * 2 * H + h] = dt;
            gates[(size_t)t * 2 * H + H + h] = -expf(a_log[h]) * dt;
        }
        return;
    }
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= C) return;
    float in[SSD_PREP_TOKENS], w[MT], x[MT];
#pragma unroll
    for (int i = 0; i < SSD_PREP_TOKENS; i++) in[i] = i < cnt ? proj[(size_t)(t0 + i) * N + x_off + c] : 0.0f;
#pragma unroll
    for (int j = 0; j < MT; j++) w[j] = j < taps ? conv_w[(size_t)c * taps + (taps - 1 - j)] : 0.0f;
    float before[MT - 1];                                   // the rows in front of the block's first token, if they are the same request's
#pragma unroll
    for (int j = 0; j < MT - 1; j++) before[j] = (j < taps - 1 && t0 - (j + 1) >= 0) ? proj[(size_t)(t0 - (j + 1)) * N + x_off + c] : 0.0f;
    const float b = conv_b ? conv_b[c] : 0.0f;
    int seg = -1;
#pragma unroll
    for (int i = 0; i < SSD_PREP_TOKENS; i++) {
        if (i < cnt) {
            const int t = t0 + i, s = token_seg[t];
            if (s != seg) {                                 // the first token here of a request: its earlier inputs
                seg = s;
                const int at = t - seg_starts[s], slot = seg_slots[s];
                const float* old = slot >= 0 ? state + (size_t)slot * state_stride + conv_off : nullptr;
#pragma unroll
                for (int j = 0; j < MT - 1; j++) {
                    x[j] = 0.0f;
                    if (j < taps - 1) {
                        const int src = at - (j + 1);
                        if (src >= 0) x[j] = before[j];     // only at the block's first token: any other that begins here is its request's first
                        else if (old) x[j] = old[(size_t)(taps - 1 + src) * C + c];
                    }
                }
            }
            float acc = b;
#pragma unroll
            for (int j = MT - 1; j >= 1; j--)
                if (j < taps) acc = fmaf(w[j], x[j - 1], acc);
            acc = fmaf(w[0], in[i], acc);
            xbc[(size_t)t * C + c] = from_f32<T>(silu_f(acc));
#pragma unroll
            for (int j = MT - 2; j >= 1; j--) x[j] = x[j - 1];
            if (MT > 1) x[0] = in[i];
        }
    }
}

// A stage: B [chunk][DP] | C [chunk][DP] | x [chunk][16] | dt [chunk] | decay [chunk]
__host__ __device__ constexpr int ssd_stage_floats(int DPT) { return SSD_CHUNK * (2 * 8 * DPT + 16 + 2); }

// The eight lanes of a column: lane group g has rows 32 j + 4 g .. + 3.
template <typename T, int DPT>
__global__ void __launch_bounds__(SSD_THREADS) ssd_recurrence_kernel(const T* __restrict__ xbc, const float* __restrict__ gates,
                                                                     const float* __restrict__ D, const int32_t* __restrict__ seg_starts,
                                                                     const int32_t* __restrict__ seg_slots, float* __restrict__ state, size_t state_stride,
                                                                     float* __restrict__ y, int C, int H, int G, int N, int P) {
    constexpr int DP = 8 * DPT, COLS = 16, STAGE = ssd_stage_floats(DPT);
    extern __shared__ __align__(16) float ssd_sm[];
    dependency_wait();
    let_dependents_start();
    const int seg = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int rg = lane >> 2, cl = warp * 4 + (lane & 3);
    const int col0 = blockIdx.x * COLS, col = col0 + cl;
    const int first = seg_starts[seg], end = seg_starts[seg + 1], slot = seg_slots[seg];
    if (first >= end) return;
    const int g = h / (H / G);
    const int x_off = h * P + col0, b_off = H * P + g * N, c_off = H * P + G * N + g * N;
    float* st = (slot >= 0 && col < P) ? state + (size_t)slot * state_stride + (size_t)h * N * P + col : nullptr;
    float S[DPT];
#pragma unroll
    for (int j = 0; j < DPT; j++) {
        const int d = 32 * (j >> 2) + 4 * rg + (j & 3);
        S[j] = (st && d < N) ? st[(size_t)d * P] : 0.0f;
    }
    const float dd = D[h];
    auto stage = [&](int chunk) {
        float* sb = ssd_sm + (chunk & 1) * STAGE;
        float* sc = sb + SSD_CHUNK * DP;
        float* sx = sc + SSD_CHUNK * DP;
        float* sd = sx + SSD_CHUNK * COLS;
        float* sa = sd + SSD_CHUNK;
        const int t0 = first + chunk * SSD_CHUNK, cnt = min(SSD_CHUNK, end - t0);
        for (int t = warp; t < cnt; t += SSD_THREADS / 32) {
            const T* row = xbc + (size_t)(t0 + t) * C;
            for (int d = lane; d < DP; d += 32) {
                sb[t * DP + d] = d < N ? to_f32<T>(row[b_off + d]) : 0.0f;
                sc[t * DP + d] = d < N ? to_f32<T>(row[c_off + d]) : 0.0f;
            }
            if (lane < COLS) sx[t * COLS + lane] = col0 + lane < P ? to_f32<T>(row[x_off + lane]) : 0.0f;
            if (lane == 0) sd[t] = gates[(size_t)(t0 + t) * 2 * H + h];
            if (lane == 1) sa[t] = expf(gates[(size_t)(t0 + t) * 2 * H + H + h]);
        }
    };
    const int chunks = (end - first + SSD_CHUNK - 1) / SSD_CHUNK;
    stage(0);
    for (int c = 0; c < chunks; c++) {
        __syncthreads();                                    // this stage is written, and the other one was read a round ago
        if (c + 1 < chunks) stage(c + 1);
        const float* sb = ssd_sm + (c & 1) * STAGE;
        const float* sc = sb + SSD_CHUNK * DP;
        const float* sx = sc + SSD_CHUNK * DP;
        const float* sd = sx + SSD_CHUNK * COLS;
        const float* sa = sd + SSD_CHUNK;
        const int t0 = first + c * SSD_CHUNK, cnt = min(SSD_CHUNK, end - t0);
        for (int t = 0; t < cnt; t++) {
            const float xx = sx[t * COLS + cl], u = sd[t] * xx, a = sa[t];
            const float4* b4 = reinterpret_cast<const float4*>(sb + t * DP) + rg;
            const float4* c4 = reinterpret_cast<const float4*>(sc + t * DP) + rg;
            float p = 0.0f;
#pragma unroll
            for (int j = 0; j < DPT / 4; j++) {
                const float4 bb = b4[8 * j], cc = c4[8 * j];
                S[4 * j + 0] = fmaf(bb.x, u, a * S[4 * j + 0]);
                S[4 * j + 1] = fmaf(bb.y, u, a * S[4 * j + 1]);
                S[4 * j + 2] = fmaf(bb.z, u, a * S[4 * j + 2]);
                S[4 * j + 3] = fmaf(bb.w, u, a * S[4 * j + 3]);
                p = fmaf(S[4 * j + 0], cc.x, p);
                p = fmaf(S[4 * j + 1], cc.y, p);
                p = fmaf(S[4 * j + 2], cc.z, p);
                p = fmaf(S[4 * j + 3], cc.w, p);
            }
#pragma unroll
            for (int off = 4; off < 32; off <<= 1) p += __shfl_xor_sync(0xffffffffu, p, off);
            if (rg == 0 && col < P) y[((size_t)(t0 + t) * H + h) * P + col] = fmaf(dd, xx, p);
        }
    }
    if (!st) return;
#pragma unroll
    for (int j = 0; j < DPT; j++) {
        const int d = 32 * (j >> 2) + 4 * rg + (j & 3);
        if (d < N) st[(size_t)d * P] = S[j];
    }
}

template <int V> struct SsdVec;
template <> struct SsdVec<1> { typedef float type; };
template <> struct SsdVec<4> { typedef float4 type; };

// A thread holds V neighbouring columns of up to J rows (rows ry, ry + 16, ...); 16 threads side by side cover 16 V columns.
template <typename T, int V, int J>
__global__ void __launch_bounds__(256) ssd_decode_kernel(const float* __restrict__ proj, int N_proj, int x_off, int dt_off,
                                                         const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                                                         const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ D,
                                                         const int32_t* __restrict__ seg_starts, const int32_t* __restrict__ seg_slots,
                                                         float* __restrict__ state, size_t state_stride, size_t conv_off, float* __restrict__ y, int C,
                                                         int H, int G, int N, int P, int taps) {
    constexpr int COLS = 16 * V;
    typedef typename SsdVec<V>::type vec_t;
    __shared__ float sbc[2 * 16 * J], sx[COLS], red[8 * COLS];
    const int seg = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, cx = tid & 15, ry = tid >> 4;
    const int col0 = blockIdx.x * COLS, col = col0 + cx * V;
    const int t = seg_starts[seg], slot = seg_slots[seg];
    const bool any = t < seg_starts[seg + 1];
    float* row = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
    float* st = (row && col < P) ? row + (size_t)h * N * P + col : nullptr;     // V = 4: P is a multiple of four
    // the kernel before this one writes neither the states nor the weights: their values are asked for before the wait
    float S[J][V];
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int d = ry + 16 * j;
        if (any && st && d < N) {
            *reinterpret_cast<vec_t*>(S[j]) = *reinterpret_cast<const vec_t*>(st + (size_t)d * P);
        } else {
#pragma unroll
            for (int v = 0; v < V; v++) S[j][v] = 0.0f;
        }
    }
    const float A = -expf(a_log[h]), dtb = dt_bias[h], dd = D[h];
    dependency_wait();
    let_dependents_start();
    if (!any) return;
    const int g = h / (H / G);
    const float* in = proj + (size_t)t * N_proj;
    const float dt_raw = in[dt_off + h];
    for (int i = tid; i < 2 * N + COLS; i += 256) {         // B and C of the head's group, x of the block's columns
        int c;
        if (i < N) c = H * P + g * N + i;
        else if (i < 2 * N) c = H * P + G * N + g * N + (i - N);
        else { if (col0 + i - 2 * N >= P) { sx[i - 2 * N] = 0.0f; continue; } c = h * P + col0 + (i - 2 * N); }
        float acc = conv_b ? conv_b[c] : 0.0f;
        for (int j = taps - 1; j >= 1; j--)
            if (row) acc = fmaf(conv_w[(size_t)c * taps + (taps - 1 - j)], row[conv_off + (size_t)(taps - 1 - j) * C + c], acc);
        acc = fmaf(conv_w[(size_t)c * taps + taps - 1], in[x_off + c], acc);
        const float v = to_f32<T>(from_f32<T>(silu_f(acc)));
        if (i < N) sbc[i] = v;
        else if (i < 2 * N) sbc[16 * J + i - N] = v;
        else sx[i - 2 * N] = v;
    }
    const float dt = softplus_f(dt_raw + dtb), a = expf(A * dt);
    __syncthreads();
    float u[V], p[V];
#pragma unroll
    for (int v = 0; v < V; v++) { u[v] = dt * sx[cx * V + v]; p[v] = 0.0f; }
#pragma unroll
    for (int j = 0; j < J; j++) {
        const int d = ry + 16 * j;
        if (d < N) {
            const float b = sbc[d], cc = sbc[16 * J + d];
#pragma unroll
            for (int v = 0; v < V; v++) {
                S[j][v] = fmaf(b, u[v], a * S[j][v]);
                p[v] = fmaf(S[j][v], cc, p[v]);
            }
            if (st) *reinterpret_cast<vec_t*>(st + (size_t)d * P) = *reinterpret_cast<const vec_t*>(S[j]);
        }
    }
#pragma unroll
    for (int v = 0; v < V; v++) p[v] += __shfl_xor_sync(0xffffffffu, p[v], 16);     // the two row groups of a warp
    if ((tid & 31) < 16) {
#pragma unroll
        for (int v = 0; v < V; v++) red[(tid >> 5) * COLS + cx * V + v] = p[v];
    }
    __syncthreads();
    if (tid < COLS && col0 + tid < P) {
        float s = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; w++) s += red[w * COLS + tid];
        y[((size_t)t * H + h) * P + col0 + tid] = fmaf(dd, sx[tid], s);
    }
}

template <typename T> __device__ __forceinline__ void ssd_store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void ssd_store4<float>(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void ssd_store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

template <typename T>
__global__ void __launch_bounds__(256) ssd_gate_kernel(const float* __restrict__ y, const float* __restrict__ proj, int N, int z_off, int x_off,
                                                       const float* __restrict__ w, float eps, float mult, int inner, int parts, T* __restrict__ out,
                                                       int out_ld, const int32_t* __restrict__ seg_starts, const int32_t* __restrict__ seg_slots,
                                                       float* __restrict__ state, size_t state_stride, size_t conv_off, int C, int taps, int vec, int tokens) {
    extern __shared__ __align__(16) float sg_sm[];          // [inner] gated values, [parts] 1 / rms
    __shared__ float scratch[32];
    float* inv = sg_sm + inner;
    dependency_wait();
    let_dependents_start();
    if (blockIdx.x >= tokens) {                             // the convolution's memory: a thread a channel of a segment
        const int per = (C + 255) / 256, seg = (blockIdx.x - tokens) / per, c = (blockIdx.x - tokens) % per * 256 + threadIdx.x;
        const int first = seg_starts[seg], n = seg_starts[seg + 1] - first, slot = seg_slots[seg];
        if (slot < 0 || n <= 0 || c >= C) return;
        float* mem = state + (size_t)slot * state_stride + conv_off + c;
        float v[DR_MAX_TAPS];                               // the last taps - 1 inputs, of which a short step leaves some of the old ones
#pragma unroll
        for (int j = 0; j < DR_MAX_TAPS; j++)
            if (j < taps - 1) {
                const int src = n - (taps - 1) + j;
                v[j] = src >= 0 ? proj[(size_t)(first + src) * N + x_off + c] : mem[(size_t)(j + n) * C];
            }
#pragma unroll
        for (int j = 0; j < DR_MAX_TAPS; j++)
            if (j < taps - 1) mem[(size_t)j * C] = v[j];
        return;
    }
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const float* in = proj + (size_t)t * N;
    if (vec) {
        for (int i = tid * 4; i < inner; i += 1024) {
            const float4 a = *reinterpret_cast<const float4*>(y + (size_t)t * inner + i), z = *reinterpret_cast<const float4*>(in + z_off + i);
            *reinterpret_cast<float4*>(sg_sm + i) = make_float4(a.x * silu_f(z.x), a.y * silu_f(z.y), a.z * silu_f(z.z), a.w * silu_f(z.w));
        }
    } else {
        for (int i = tid; i < inner; i += 256) sg_sm[i] = y[(size_t)t * inner + i] * silu_f(in[z_off + i]);
    }
    const int size = inner / parts;
    __syncthreads();
    if (parts >= 8) {
        for (int p = warp; p < parts; p += 8) {
            float ss = 0.0f;
            for (int i = lane; i < size; i += 32) ss = fmaf(sg_sm[p * size + i], sg_sm[p * size + i], ss);
            ss = warp_sum(ss);
            if (lane == 0) inv[p] = mult / sqrtf(ss / (float)size + eps);
        }
    } else {
        for (int p = 0; p < parts; p++) {
            float ss = 0.0f;
            for (int i = tid; i < size; i += 256) ss = fmaf(sg_sm[p * size + i], sg_sm[p * size + i], ss);
            ss = block_sum(ss, scratch);
            if (tid == 0) inv[p] = mult / sqrtf(ss / (float)size + eps);
        }
    }
    __syncthreads();
    T* dst = out + (size_t)t * out_ld;
    if (vec && size % 4 == 0) {
        for (int i = tid * 4; i < inner; i += 1024) {
            const float4 a = *reinterpret_cast<const float4*>(sg_sm + i), ww = *reinterpret_cast<const float4*>(w + i);
            const float r = inv[i / size];
            ssd_store4<T>(dst + i, (a.x * r) * ww.x, (a.y * r) * ww.y, (a.z * r) * ww.z, (a.w * r) * ww.w);
        }
    } else {
        for (int i = tid; i < inner; i += 256) dst[i] = from_f32<T>((sg_sm[i] * inv[i / size]) * w[i]);
    }
}

template <typename... KArgs, typename... Args>
static int ssd_launch(bool few, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
    return few ? launch_dependent(kernel, grid, block, smem, stream, args...) : launch_plain(kernel, grid, block, smem, stream, args...);
}

}  // namespace vk

using namespace vk;

VK_API int vk_ssd_max_state() { return 256; }
VK_API int vk_ssd_max_taps() { return DR_MAX_TAPS; }

static bool ssd_sizes_ok(int H, int G, int N, int P, int taps) {
    return H > 0 && G > 0 && H % G == 0 && N > 0 && P > 0 && taps > 0 && N <= 256 && taps <= DR_MAX_TAPS && H <= 65535;
}

// proj float32 [tokens][N_proj] with the channels x | B | C (C of them) at x_off and the step sizes at dt_off; conv_w float32 [C][taps], conv_b
// [C] or null; xbc [tokens][C] in dtype; gates float32 [tokens][2 H].
VK_API int vk_ssd_prepare(const float* proj, int N_proj, int x_off, int dt_off, const float* conv_w, const float* conv_b, const float* dt_bias,
                          const float* a_log, const int32_t* token_seg, const int32_t* seg_starts, const int32_t* seg_slots, const float* state,
                          size_t state_stride, void* xbc, float* gates, int tokens, int H, int G, int N, int P, int taps, int dtype,
                          cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    const int C = H * P + 2 * G * N;
    if (!ssd_sizes_ok(H, G, N, P, taps) || x_off < 0 || dt_off < 0 || x_off + C > N_proj || dt_off + H > N_proj) return VK_BAD_SHAPE;
    dim3 grid((tokens + SSD_PREP_TOKENS - 1) / SSD_PREP_TOKENS, (C + 255) / 256 + 1);
    const bool few = tokens <= DR_DEPENDENT_TOKENS;
    const size_t conv_off = (size_t)H * N * P;
#define VK_SSDP(T, MT)                                                                                                                       \
    return ssd_launch(few, ssd_prepare_kernel<T, MT>, grid, dim3(256), 0, stream, proj, N_proj, x_off, dt_off, conv_w, conv_b, dt_bias, a_log, \
                      token_seg, seg_starts, seg_slots, state, state_stride, conv_off, (T*)xbc, gates, C, H, taps, tokens)
    if (dtype == 0) {
        if (taps <= 4) VK_SSDP(float, 4);
        VK_SSDP(float, DR_MAX_TAPS);
    }
    if (taps <= 4) VK_SSDP(__nv_bfloat16, 4);
    VK_SSDP(__nv_bfloat16, DR_MAX_TAPS);
#undef VK_SSDP
}

// xbc [tokens][C] in dtype and gates as ssd_prepare writes them; y float32 [tokens][H P].
VK_API int vk_ssd_recurrence(const void* xbc, const float* gates, const float* D, const int32_t* seg_starts, const int32_t* seg_slots, float* state,
                             size_t state_stride, float* y, int segments, int H, int G, int N, int P, int dtype, cudaStream_t stream) {
    if (segments <= 0) return VK_OK;
    if (!ssd_sizes_ok(H, G, N, P, 1)) return VK_BAD_SHAPE;
    if (segments > 65535) return VK_TOO_LARGE;
    const int C = H * P + 2 * G * N;
    dim3 grid((P + 15) / 16, H, segments);
#define VK_SSDR(T, DPT)                                                                                                                       \
    do {                                                                                                                                      \
        auto kern = ssd_recurrence_kernel<T, DPT>;                                                                                            \
        const size_t smem = 2 * (size_t)ssd_stage_floats(DPT) * sizeof(float);                                                                \
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                                   \
        if (e != cudaSuccess) return (int)e;                                                                                                  \
        return launch_plain(kern, grid, dim3(SSD_THREADS), smem, stream, (const T*)xbc, gates, D, seg_starts, seg_slots, state, state_stride, \
                            y, C, H, G, N, P);                                                                                                \
    } while (0)
    if (dtype == 0) {
        if (N <= 32) VK_SSDR(float, 4);
        if (N <= 64) VK_SSDR(float, 8);
        if (N <= 128) VK_SSDR(float, 16);
        VK_SSDR(float, 32);
    }
    if (N <= 32) VK_SSDR(__nv_bfloat16, 4);
    if (N <= 64) VK_SSDR(__nv_bfloat16, 8);
    if (N <= 128) VK_SSDR(__nv_bfloat16, 16);
    VK_SSDR(__nv_bfloat16, 32);
#undef VK_SSDR
}

// Every segment is one token: convolution, gates, one step and the state's update in one launch (the convolution's memory is left to
// ssd_gate).  dtype: what the convolution's results are rounded to.
VK_API int vk_ssd_decode(const float* proj, int N_proj, int x_off, int dt_off, const float* conv_w, const float* conv_b, const float* dt_bias,
                         const float* a_log, const float* D, const int32_t* seg_starts, const int32_t* seg_slots, float* state, size_t state_stride,
                         float* y, int segments, int H, int G, int N, int P, int taps, int dtype, cudaStream_t stream) {
    if (segments <= 0) return VK_OK;
    const int C = H * P + 2 * G * N;
    if (!ssd_sizes_ok(H, G, N, P, taps) || x_off < 0 || dt_off < 0 || x_off + C > N_proj || dt_off + H > N_proj) return VK_BAD_SHAPE;
    if (segments > 65535) return VK_TOO_LARGE;
    const bool vec = P % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
    const size_t conv_off = (size_t)H * N * P;
    dim3 grid(vec ? (P + 63) / 64 : (P + 15) / 16, H, segments);
#define VK_SSDD(T, V, J)                                                                                                                       \
    return launch_dependent(ssd_decode_kernel<T, V, J>, grid, dim3(256), 0, stream, proj, N_proj, x_off, dt_off, conv_w, conv_b, dt_bias, a_log, \
                            D, seg_starts, seg_slots, state, state_stride, conv_off, y, C, H, G, N, P, taps)
#define VK_SSDDJ(T, V)                 \
    do {                               \
        if (N <= 64) VK_SSDD(T, V, 4); \
        if (N <= 128) VK_SSDD(T, V, 8);\
        VK_SSDD(T, V, 16);             \
    } while (0)
    if (dtype == 0) {
        if (vec) VK_SSDDJ(float, 4);
        VK_SSDDJ(float, 1);
    }
    if (vec) VK_SSDDJ(__nv_bfloat16, 4);
    VK_SSDDJ(__nv_bfloat16, 1);
#undef VK_SSDDJ
#undef VK_SSDD
}

// out (rows out_ld apart, H P columns each) in dtype = mult * rms-normed (in `parts` equal parts) (y silu(z)) * w; moves the convolution's
// memory of every segment on.
VK_API int vk_ssd_gate(const float* y, const float* proj, int N_proj, int z_off, int x_off, const float* w, float eps, float mult, int parts, void* out,
                       int out_ld, const int32_t* seg_starts, const int32_t* seg_slots, int segments, float* state, size_t state_stride, int tokens, int H, int G, int N, int P, int taps, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    const int C = H * P + 2 * G * N, inner = H * P;
    if (!ssd_sizes_ok(H, G, N, P, taps) || parts <= 0 || inner % parts || z_off < 0 || z_off + inner > N_proj || x_off < 0 || x_off + C > N_proj ||
        out_ld < inner)
        return VK_BAD_SHAPE;
    const size_t smem = (size_t)(inner + parts) * sizeof(float);
    if (smem > 200 * 1024) return VK_TOO_LARGE;
    const bool few = tokens <= DR_DEPENDENT_TOKENS;
    const size_t conv_off = (size_t)H * N * P;
    const int vec = inner % 4 == 0 && N_proj % 4 == 0 && z_off % 4 == 0 && out_ld % 4 == 0 && ((uintptr_t)y % 16) == 0 && ((uintptr_t)proj % 16) == 0 &&
                    ((uintptr_t)w % 16) == 0 && ((uintptr_t)out % (dtype == 0 ? 16 : 8)) == 0;
    const dim3 grid(tokens + (taps > 1 ? segments * ((C + 255) / 256) : 0));
#define VK_SSDG(T)                                                                                                                           \
    do {                                                                                                                                     \
        auto kern = ssd_gate_kernel<T>;                                                                                                      \
        if (smem > 48 * 1024) {                                                                                                              \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                              \
            if (e != cudaSuccess) return (int)e;                                                                                             \
        }                                                                                                                                    \
        return ssd_launch(few, kern, grid, dim3(256), smem, stream, y, proj, N_proj, z_off, x_off, w, eps, mult, inner, parts, (T*)out, \
                          out_ld, seg_starts, seg_slots, state, state_stride, conv_off, C, taps, vec, tokens);                               \
    } while (0)
    if (dtype == 0) VK_SSDG(float);
    VK_SSDG(__nv_bfloat16);
#undef VK_SSDG
}
