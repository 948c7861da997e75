// The state-space mixer's recurrence in chunks of 64 tokens on the tensor cores (bfloat16; ssd.cu states the recurrence).
//
// With l_t the log decay of token t of a chunk and L_t = l_1 + .. + l_t, S the state before the chunk:
//
//     y_t = e^(L_t) S^T C_t + sum_(i <= t) e^(L_t - L_i) dt_i (C_t . B_i) x_i + D x_t
//     S'  = e^(L_64) S + sum_i e^(L_64 - L_i) dt_i B_i x_i^T
//
//  ssd_chunk_state  what a chunk adds to the state, all chunks side by side: B^T (w x), w_i = e^(L_last - L_i) dt_i.
//  ssd_chunk_scan   the states before every chunk, a thread a few elements of a head's state, a request's chunks in order; the request's
//                   own state is read before its first chunk and written after its last.
//  ssd_chunk_out    the outputs, all chunks side by side: C B^T, its causal weights, their product with x, and C S.
//
// B, C and x are bfloat16 as the convolution leaves them.  What is float32 in the recurrence (weights, states) goes into a product as a
// high and a low bfloat16 part, so that only B, C and x are 16-bit quantities; every exponent is at most 0; sums are float32.  A chunk
// begins at a request's first token of the step.  The products are small (64 rows, 64 columns of a head's values): mma.sync with two
// to three blocks a multiprocessor; a tile of tcgen05 (128 rows) would be half empty.
//
// Which chunk a block has is worked out from the segments' starts on the device, so the launches depend on the step's counts alone.
#include "delta_common.cuh"

namespace vk {

constexpr int SC_Q = 64;                // tokens of a chunk
constexpr int SC_P = 64;                // columns of a head's values a block takes
constexpr int SC_THREADS = 128;
constexpr int SC_LD = SC_P + 8;         // a padded row of 64 values: 16-byte shifts keep ldmatrix free of bank conflicts

__device__ __forceinline__ void sc_ldsm4(uint32_t* r, const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_ldsm4t(uint32_t* r, const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void sc_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t sc_pack(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
// the parts that rounding (a, b) to bfloat16 leaves over, again in bfloat16
__device__ __forceinline__ uint32_t sc_pack_rest(float a, float b, uint32_t hi) {
    return sc_pack(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

struct SscChunk { int seg, first, rows; };      // segment (-1: this block has no chunk), first token, rows

// The chunk with number n: segments have ceil(length / 64) chunks each, numbered one after another.
__device__ __forceinline__ SscChunk ssc_find(int n, const int32_t* __restrict__ seg_starts, int segments, int* sh) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        int base = 0, found = 0;
        for (int s0 = 0; s0 < segments && !found; s0 += 32) {
            const int s = s0 + lane;
            const int a = s < segments ? seg_starts[s] : 0, b = s < segments ? seg_starts[s + 1] : 0;
            const int mine = (b - a + SC_Q - 1) / SC_Q;
            int upto = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, upto, o);
                if (lane >= o) upto += v;
            }
            const int lo = base + upto - mine;
            const bool here = n >= lo && n < lo + mine;
            if (here) {
                sh[0] = s;
                sh[1] = a + (n - lo) * SC_Q;
                sh[2] = min(SC_Q, b - sh[1]);
            }
            found = __any_sync(0xffffffffu, here);
            base += __shfl_sync(0xffffffffu, upto, 31);
        }
        if (!found && lane == 0) sh[0] = -1;
    }
    __syncthreads();
    return SscChunk{sh[0], sh[1], sh[2]};
}

// rows x cols bfloat16 from src (rows ld apart) into dst (rows COLS + 8 apart), zeros up to ROWS x COLS (COLS a multiple of 8)
template <int ROWS, int COLS>
__device__ __forceinline__ void ssc_tile(__nv_bfloat16* dst, const __nv_bfloat16* __restrict__ src, size_t ld, int rows, int cols) {
    const bool vec = (reinterpret_cast<uintptr_t>(src) % 16 == 0) && ld % 8 == 0 && cols % 8 == 0;
    constexpr int PIECES = COLS / 8;
#pragma unroll 4
    for (int i = threadIdx.x; i < ROWS * PIECES; i += SC_THREADS) {
        const int r = i / PIECES, c = (i % PIECES) * 8;
        __nv_bfloat16* d = dst + r * (COLS + 8) + c;
        if (r < rows && c < cols && vec) {
            dr_cp_async16(d, src + r * ld + c);
        } else {
            uint32_t v[4];
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int c0 = c + 2 * e;
                const __nv_bfloat16 z = __float2bfloat16_rn(0.0f);
                const __nv_bfloat162 two = __halves2bfloat162(r < rows && c0 < cols ? src[r * ld + c0] : z, r < rows && c0 + 1 < cols ? src[r * ld + c0 + 1] : z);
                v[e] = *reinterpret_cast<const uint32_t*>(&two);
            }
            *reinterpret_cast<uint4*>(d) = make_uint4(v[0], v[1], v[2], v[3]);
        }
    }
}

// L (sums of the log decays up to and with each token) and dt of the chunk's tokens; beyond the last token nothing decays and dt is 0.
__device__ __forceinline__ void ssc_gates(float* L, float* dt, const float* __restrict__ gates, int first, int rows, int H, int h) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        float carry = 0.0f;
#pragma unroll
        for (int k = 0; k < SC_Q / 32; k++) {
            const int i = k * 32 + lane;
            const float* p = gates + (size_t)(first + i) * 2 * H + h;
            float s = i < rows ? p[H] : 0.0f;
            dt[i] = i < rows ? p[0] : 0.0f;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += v;
            }
            L[i] = carry + s;
            carry += __shfl_sync(0xffffffffu, s, 31);
        }
    }
}

// NP: the state's rows, rounded up to a size that is built
template <int NP>
__global__ void __launch_bounds__(SC_THREADS) ssd_chunk_state_kernel(const __nv_bfloat16* __restrict__ xbc, const float* __restrict__ gates,
                                                                     const int32_t* __restrict__ seg_starts, int segments, float* __restrict__ add,
                                                                     float* __restrict__ whole, int C, int H, int G, int N, int P) {
    extern __shared__ __align__(16) unsigned char ss_raw[];
    __shared__ float L[SC_Q], dt[SC_Q];
    __shared__ int find[3];
    constexpr int LDB = NP + 8;
    __nv_bfloat16* sb = reinterpret_cast<__nv_bfloat16*>(ss_raw);       // [64][LDB]
    __nv_bfloat16* sx = sb + SC_Q * LDB;                                // [64][SC_LD] high parts of w x (first: x itself)
    __nv_bfloat16* sl = sx + SC_Q * SC_LD;                              // [64][SC_LD] low parts
    const SscChunk ch = ssc_find(blockIdx.x, seg_starts, segments, find);
    if (ch.seg < 0) return;
    const int h = blockIdx.y, p0 = blockIdx.z * SC_P, pc = min(SC_P, P - p0), g = h / (H / G);
    const __nv_bfloat16* base = xbc + (size_t)ch.first * C;
    ssc_tile<SC_Q, NP>(sb, base + H * P + g * N, C, ch.rows, N);
    ssc_tile<SC_Q, SC_P>(sx, base + h * P + p0, C, ch.rows, pc);
    asm volatile("cp.async.commit_group;" ::: "memory");
    ssc_gates(L, dt, gates, ch.first, ch.rows, H, h);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (blockIdx.z == 0 && tid == 0) whole[(size_t)blockIdx.x * H + h] = expf(L[SC_Q - 1]);
    for (int i = tid; i < SC_Q * SC_P / 2; i += SC_THREADS) {           // w x in two parts
        const int r = i / (SC_P / 2), c = (i % (SC_P / 2)) * 2;
        const float w = expf(L[SC_Q - 1] - L[r]) * dt[r];
        const uint32_t v = *reinterpret_cast<const uint32_t*>(sx + r * SC_LD + c);
        const float a = w * __uint_as_float(v << 16), b = w * __uint_as_float(v & 0xffff0000u);
        const uint32_t hi = sc_pack(a, b);
        *reinterpret_cast<uint32_t*>(sx + r * SC_LD + c) = hi;
        *reinterpret_cast<uint32_t*>(sl + r * SC_LD + c) = sc_pack_rest(a, b, hi);
    }
    __syncthreads();
    float* out = add + ((size_t)blockIdx.x * H + h) * N * P;
    const int gid = lane >> 2, tig = lane & 3;
    for (int mt = warp; mt < NP / 16; mt += SC_THREADS / 32) {          // 16 rows of the state
        float acc[8][4];
#pragma unroll
        for (int nb = 0; nb < 8; nb++) acc[nb][0] = acc[nb][1] = acc[nb][2] = acc[nb][3] = 0.0f;
#pragma unroll
        for (int kt = 0; kt < SC_Q / 16; kt++) {
            uint32_t a[4];
            // rows of the state are columns of B: the four 8 x 8 pieces (tokens, rows) transposed on their way
            sc_ldsm4t(a, sb + (kt * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * LDB + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int nb = 0; nb < 8; nb += 2) {
                uint32_t b[4];
                const int at = (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LD + nb * 8 + (lane >> 4) * 8;
                sc_ldsm4t(b, sx + at);
                sc_mma(acc[nb], a, b[0], b[1]);
                sc_mma(acc[nb + 1], a, b[2], b[3]);
                sc_ldsm4t(b, sl + at);
                sc_mma(acc[nb], a, b[0], b[1]);
                sc_mma(acc[nb + 1], a, b[2], b[3]);
            }
        }
        const bool two = P % 2 == 0;
#pragma unroll
        for (int nb = 0; nb < 8; nb++) {
            const int c = nb * 8 + tig * 2;
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int r = mt * 16 + gid + half * 8;
                if (r >= N || c >= pc) continue;
                float* d = out + (size_t)r * P + p0 + c;
                if (two) {
                    *reinterpret_cast<float2*>(d) = make_float2(acc[nb][2 * half], acc[nb][2 * half + 1]);
                } else {
                    d[0] = acc[nb][2 * half];
                    if (c + 1 < pc) d[1] = acc[nb][2 * half + 1];
                }
            }
        }
    }
}

// E elements of a head's state a thread; the states before the chunks go out as high and low bfloat16 parts.
template <int E>
__global__ void __launch_bounds__(256) ssd_chunk_scan_kernel(const float* __restrict__ add, const float* __restrict__ whole,
                                                             const int32_t* __restrict__ seg_starts, const int32_t* __restrict__ seg_slots,
                                                             float* __restrict__ state, size_t state_stride, __nv_bfloat16* __restrict__ hi,
                                                             __nv_bfloat16* __restrict__ lo, int H, int NPe) {
    __shared__ int base_sh;
    const int seg = blockIdx.z, h = blockIdx.y;
    if (threadIdx.x < 32) {                                             // chunks of the segments before this one
        int n = 0;
        for (int s = threadIdx.x; s < seg; s += 32) n += (seg_starts[s + 1] - seg_starts[s] + SC_Q - 1) / SC_Q;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
        if (threadIdx.x == 0) base_sh = n;
    }
    __syncthreads();
    const int i = (blockIdx.x * 256 + threadIdx.x) * E;
    if (i >= NPe) return;
    const int base = base_sh, chunks = (seg_starts[seg + 1] - seg_starts[seg] + SC_Q - 1) / SC_Q, slot = seg_slots[seg];
    float* st = slot >= 0 ? state + (size_t)slot * state_stride + (size_t)h * NPe + i : nullptr;
    float s[E];
    auto load = [](float* d, const float* p) {
        if (E == 4) *reinterpret_cast<float4*>(d) = *reinterpret_cast<const float4*>(p);
        else d[0] = *p;
    };
#pragma unroll
    for (int e = 0; e < E; e++) s[e] = 0.0f;
    if (st) load(s, st);
    constexpr int AHEAD = 4;                                            // chunks whose additions are on their way together
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float v[AHEAD][E], w[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                load(v[u], add + ((size_t)(base + c0 + u) * H + h) * NPe + i);
                w[u] = whole[(size_t)(base + c0 + u) * H + h];
            }
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                const size_t at = ((size_t)(base + c0 + u) * H + h) * NPe + i;
                if (E == 4) {
                    const uint32_t h0 = sc_pack(s[0], s[1]), h1 = sc_pack(s[2], s[3]);
                    *reinterpret_cast<uint2*>(hi + at) = make_uint2(h0, h1);
                    *reinterpret_cast<uint2*>(lo + at) = make_uint2(sc_pack_rest(s[0], s[1], h0), sc_pack_rest(s[2], s[3], h1));
                } else {
                    const __nv_bfloat16 a = __float2bfloat16_rn(s[0]);
                    hi[at] = a;
                    lo[at] = __float2bfloat16_rn(s[0] - __bfloat162float(a));
                }
#pragma unroll
                for (int e = 0; e < E; e++) s[e] = fmaf(w[u], s[e], v[u][e]);
            }
    }
    if (!st) return;
    if (E == 4) *reinterpret_cast<float4*>(st) = make_float4(s[0], s[1], s[2], s[3]);
    else *st = s[0];
}

template <int NP>
__global__ void __launch_bounds__(SC_THREADS) ssd_chunk_out_kernel(const __nv_bfloat16* __restrict__ xbc, const float* __restrict__ gates,
                                                                   const float* __restrict__ D, const int32_t* __restrict__ seg_starts, int segments,
                                                                   const __nv_bfloat16* __restrict__ hi, const __nv_bfloat16* __restrict__ lo,
                                                                   float* __restrict__ y, int C, int H, int G, int N, int P) {
    extern __shared__ __align__(16) unsigned char so_raw[];
    __shared__ float L[SC_Q], dt[SC_Q];
    __shared__ int find[3];
    constexpr int LDB = NP + 8;
    __nv_bfloat16* sc = reinterpret_cast<__nv_bfloat16*>(so_raw);       // [64][LDB]
    __nv_bfloat16* sb = sc + SC_Q * LDB;                                // [64][LDB]
    __nv_bfloat16* sx = sb + SC_Q * LDB;                                // [64][SC_LD]
    __nv_bfloat16* sh = sx + SC_Q * SC_LD;                              // [NP][SC_LD] the state before the chunk, high parts
    __nv_bfloat16* sl = sh + NP * SC_LD;                                // [NP][SC_LD] low parts
    const SscChunk ch = ssc_find(blockIdx.x, seg_starts, segments, find);
    if (ch.seg < 0) return;
    const int h = blockIdx.y, p0 = blockIdx.z * SC_P, pc = min(SC_P, P - p0), g = h / (H / G);
    const __nv_bfloat16* base = xbc + (size_t)ch.first * C;
    const size_t st = ((size_t)blockIdx.x * H + h) * N * P + p0;
    ssc_tile<SC_Q, NP>(sc, base + H * P + G * N + g * N, C, ch.rows, N);
    ssc_tile<SC_Q, NP>(sb, base + H * P + g * N, C, ch.rows, N);
    ssc_tile<SC_Q, SC_P>(sx, base + h * P + p0, C, ch.rows, pc);
    ssc_tile<NP, SC_P>(sh, hi + st, P, N, pc);
    ssc_tile<NP, SC_P>(sl, lo + st, P, N, pc);
    asm volatile("cp.async.commit_group;" ::: "memory");
    ssc_gates(L, dt, gates, ch.first, ch.rows, H, h);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
    if (warp * 16 >= ch.rows) return;                                   // no token of this warp's sixteen; nobody waits for it below
    float s[8][4], o[8][4];
#pragma unroll
    for (int nb = 0; nb < 8; nb++) {
        s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.0f;
        o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
    }
#pragma unroll
    for (int kt = 0; kt < NP / 16; kt++) {
        uint32_t a[4];
        sc_ldsm4(a, sc + (warp * 16 + (lane & 15)) * LDB + kt * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int nb = 0; nb < 8; nb += 2) {
            uint32_t b[4];
            if (nb <= 2 * warp + 1) {                                   // tokens that some row of the warp sees
                sc_ldsm4(b, sb + (nb * 8 + (lane & 7) + ((lane >> 4) << 3)) * LDB + kt * 16 + ((lane >> 3) & 1) * 8);
                sc_mma(s[nb], a, b[0], b[1]);
                sc_mma(s[nb + 1], a, b[2], b[3]);
            }
            const int at = (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LD + nb * 8 + (lane >> 4) * 8;
            sc_ldsm4t(b, sh + at);
            sc_mma(o[nb], a, b[0], b[1]);
            sc_mma(o[nb + 1], a, b[2], b[3]);
            sc_ldsm4t(b, sl + at);
            sc_mma(o[nb], a, b[0], b[1]);
            sc_mma(o[nb + 1], a, b[2], b[3]);
        }
    }
    const int ra = warp * 16 + gid, rb = ra + 8;
    const float La = L[ra], Lb = L[rb];
    const float ea = expf(La), eb = expf(Lb);
#pragma unroll
    for (int nb = 0; nb < 8; nb++) { o[nb][0] *= ea; o[nb][1] *= ea; o[nb][2] *= eb; o[nb][3] *= eb; }
#pragma unroll
    for (int kk = 0; kk < 4; kk++) {                                    // sixteen tokens of the chunk
        if (kk > warp) break;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int nb = 2 * kk + half, i0 = nb * 8 + tig * 2;
            const float L0 = L[i0], L1 = L[i0 + 1], d0 = dt[i0], d1 = dt[i0 + 1];
            const float a0 = i0 <= ra ? s[nb][0] * (expf(La - L0) * d0) : 0.0f, a1 = i0 + 1 <= ra ? s[nb][1] * (expf(La - L1) * d1) : 0.0f;
            const float b0 = i0 <= rb ? s[nb][2] * (expf(Lb - L0) * d0) : 0.0f, b1 = i0 + 1 <= rb ? s[nb][3] * (expf(Lb - L1) * d1) : 0.0f;
            ph[2 * half] = sc_pack(a0, a1);
            ph[2 * half + 1] = sc_pack(b0, b1);
            pl[2 * half] = sc_pack_rest(a0, a1, ph[2 * half]);
            pl[2 * half + 1] = sc_pack_rest(b0, b1, ph[2 * half + 1]);
        }
#pragma unroll
        for (int nb = 0; nb < 8; nb += 2) {
            uint32_t b[4];
            sc_ldsm4t(b, sx + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LD + nb * 8 + (lane >> 4) * 8);
            sc_mma(o[nb], ph, b[0], b[1]);
            sc_mma(o[nb + 1], ph, b[2], b[3]);
            sc_mma(o[nb], pl, b[0], b[1]);
            sc_mma(o[nb + 1], pl, b[2], b[3]);
        }
    }
    const float dd = D[h];
    const bool two = P % 2 == 0;
#pragma unroll
    for (int nb = 0; nb < 8; nb++) {
        const int c = nb * 8 + tig * 2;
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int r = half ? rb : ra;
            if (r >= ch.rows || c >= pc) continue;
            const uint32_t x = *reinterpret_cast<const uint32_t*>(sx + r * SC_LD + c);
            const float v0 = fmaf(dd, __uint_as_float(x << 16), o[nb][2 * half]), v1 = fmaf(dd, __uint_as_float(x & 0xffff0000u), o[nb][2 * half + 1]);
            float* d = y + ((size_t)(ch.first + r) * H + h) * P + p0 + c;
            if (two) {
                *reinterpret_cast<float2*>(d) = make_float2(v0, v1);
            } else {
                d[0] = v0;
                if (c + 1 < pc) d[1] = v1;
            }
        }
    }
}

}  // namespace vk

using namespace vk;

static int ssc_chunks(int tokens, int segments) { return tokens / SC_Q + (segments < tokens ? segments : tokens); }
static size_t ssc_up(size_t b) { return (b + 255) / 256 * 256; }
static int ssc_rows(int N) { return N <= 16 ? 16 : N <= 32 ? 32 : N <= 64 ? 64 : N <= 128 ? 128 : 256; }     // the sizes that are built
static size_t ssc_state_smem(int NP) { return (size_t)(SC_Q * (NP + 8) + 2 * SC_Q * SC_LD) * 2; }
static size_t ssc_out_smem(int NP) { return (size_t)(2 * SC_Q * (NP + 8) + SC_Q * SC_LD + 2 * NP * SC_LD) * 2; }

VK_API size_t vk_ssd_chunked_scratch_bytes(int tokens, int segments, int H, int N, int P) {
    const size_t chunks = ssc_chunks(tokens, segments), states = chunks * H * N * P;
    return ssc_up(states * 4) + 2 * ssc_up(states * 2) + ssc_up(chunks * H * 4);
}

// xbc bfloat16 [tokens][H P + 2 G N] and gates float32 [tokens][2 H] as ssd_prepare writes them; y float32 [tokens][H P]; three kernels.
VK_API int vk_ssd_chunked(const void* xbc, const float* gates, const float* D, const int32_t* seg_starts, const int32_t* seg_slots, float* state,
                          size_t state_stride, float* y, void* scratch, int segments, int tokens, int H, int G, int N, int P, cudaStream_t stream) {
    if (segments <= 0 || tokens <= 0) return VK_OK;
    if (H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0) return VK_BAD_SHAPE;
    if (N > 256 || H > 65535 || segments > 65535) return VK_TOO_LARGE;
    if (((uintptr_t)scratch % 16) || ((uintptr_t)xbc % 4)) return VK_BAD_ALIGNMENT;
    const int chunks = ssc_chunks(tokens, segments), C = H * P + 2 * G * N;
    const size_t states = (size_t)chunks * H * N * P;
    float* add = (float*)scratch;
    __nv_bfloat16* hi = (__nv_bfloat16*)((char*)scratch + ssc_up(states * 4));
    __nv_bfloat16* lo = (__nv_bfloat16*)((char*)hi + ssc_up(states * 2));
    float* whole = (float*)((char*)lo + ssc_up(states * 2));
    dim3 grid(chunks, H, (P + SC_P - 1) / SC_P);
    const int NP = ssc_rows(N);
    const size_t smem1 = ssc_state_smem(NP), smem3 = ssc_out_smem(NP);
    auto state_kernel = NP == 16 ? ssd_chunk_state_kernel<16> : NP == 32 ? ssd_chunk_state_kernel<32> : NP == 64 ? ssd_chunk_state_kernel<64>
                      : NP == 128 ? ssd_chunk_state_kernel<128> : ssd_chunk_state_kernel<256>;
    auto out_kernel = NP == 16 ? ssd_chunk_out_kernel<16> : NP == 32 ? ssd_chunk_out_kernel<32> : NP == 64 ? ssd_chunk_out_kernel<64>
                    : NP == 128 ? ssd_chunk_out_kernel<128> : ssd_chunk_out_kernel<256>;
    cudaError_t e = cudaFuncSetAttribute(state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
    if (e != cudaSuccess) return (int)e;
    int s = launch_plain(state_kernel, grid, dim3(SC_THREADS), smem1, stream, (const __nv_bfloat16*)xbc, gates, seg_starts, segments, add, whole, C, H, G, N, P);
    if (s != VK_OK) return s;
    const int NPe = N * P;
    if (NPe % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0)
        s = launch_plain(ssd_chunk_scan_kernel<4>, dim3((NPe + 1023) / 1024, H, segments), dim3(256), 0, stream, add, whole, seg_starts, seg_slots, state,
                         state_stride, hi, lo, H, NPe);
    else
        s = launch_plain(ssd_chunk_scan_kernel<1>, dim3((NPe + 255) / 256, H, segments), dim3(256), 0, stream, add, whole, seg_starts, seg_slots, state,
                         state_stride, hi, lo, H, NPe);
    if (s != VK_OK) return s;
    return launch_plain(out_kernel, grid, dim3(SC_THREADS), smem3, stream, (const __nv_bfloat16*)xbc, gates, D, seg_starts, segments, hi, lo, y, C,
                        H, G, N, P);
}
