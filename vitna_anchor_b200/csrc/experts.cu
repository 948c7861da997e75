// A routed feed-forward: every token uses `top` of E small feed-forward layers (gated or not), with weights from a router or a table.
//
//  experts_route     one block a token: logits z = W_r x + b in float32 (a warp a logit), the `top` largest (of equal logits the lower
//                    index), weights = softmax over the chosen logits alone.  Writes ids [tokens][top] and weights [tokens][top].
//  experts_route_scored  scores s = softmax(W_r x) over experts AND identities; a token's choice goes by s + correction: of `count` equal
//                    groups of neighbours only the `keep` with the largest choice score take part, and of their members the `top` with the
//                    largest (of equals the lower index); weights s / (sum of the chosen s + 1e-20) times scale.  An id of E or more
//                    is an identity: its output is the token's input row.  The other form has a sigmoid for every score and takes the
//                    chosen scores as they are, times scale (without a correction the logits choose: a sigmoid that has rounded
//                    to 1 does not make a tie); squared, if asked: where the weight multiplies the INPUT of an expert whose
//                    activation is homogeneous of degree 2, f(s z) = s^2 f(z), its square multiplies the output.
//  experts_route_table  ids[token][k] = table[token id][k], every weight 1 / top: the experts of a token are a function of its id.
//  experts_gate_up   act[token, k] = f(W_gate,e x) * (W_up,e x) for the token's k-th expert e; a warp an output column, the token's row
//                    in shared memory.  f is one of the epilogues' activations.  Ungated: act[token, k] = f(W_up,e x).
//  experts_down      y[token] += sum_k weight_k W_down,e_k act[token, k], the experts of a token summed in the order of its list, so
//                    that the sum does not depend on what else is in the batch.
//
//  experts_shared_up, experts_shared_down   the same two for a few tokens that share experts: a block an expert and some columns, which reads its rows
//                    of the weights once for all of the step's (token, k) pairs that chose the expert (in passes of up to four pairs whose
//                    input rows lie in shared memory); the second leaves a float32 row a pair (or, where a token has one expert, adds it
//                    to y) and experts_combine adds them up.  The sums run in the order of the two kernels above, so that the
//                    result is the same bits.
//
// For a prompt's portion in bfloat16 the experts' products run on the tensor cores as products of row groups (linear_tcgen05.cu):
//  experts_sort      one block: counts the copies a group (an expert) gets, gives every group whole tiles of 128 rows one after another,
//                    and writes for each (token, k) its row, for each row its token (-1: a fill row), for each tile its group
//                    (-1: unused).  Which copy of a group gets which of its rows is left to the order of arrival: a row's product
//                    does not depend on where in a tile it stands.
//  experts_gather    a block a row: the token's input row is copied to its row of the grouped matrix.
//  experts_combine   a block a token: y[token] += sum_k weight_k out[row of (token, k)], in the order of the token's list.
//
// Nothing here comes to the host: which experts run is read by the kernels from the ids on the device, so a captured graph
// replays the part for any batch.  Products accumulate in float32 (fmaf); storage is float32 or bfloat16.
#include "common.cuh"

namespace vk {

template <typename T>
__global__ void __launch_bounds__(128) experts_route_kernel(const T* __restrict__ x, int width, const float* __restrict__ wr,
                                                            const float* __restrict__ br, int E, int top, int32_t* __restrict__ ids,
                                                            float* __restrict__ wts) {
    extern __shared__ float z[];                        // [E]
    dependency_wait();
    let_dependents_start();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const T* row = x + (size_t)t * width;
    for (int e = warp; e < E; e += nwarps) {
        const float* w = wr + (size_t)e * width;
        float acc = 0.0f;
        for (int i = lane; i < width; i += 32) acc = fmaf(to_f32<T>(row[i]), w[i], acc);
        acc = warp_sum(acc);
        if (lane == 0) z[e] = acc + (br ? br[e] : 0.0f);
    }
    __syncthreads();
    if (warp != 0) return;
    // the warp picks the largest logit `top` times; every lane knows each pick, lane k keeps the k-th weight
    __shared__ int picked[32];
    float zmax = 0.0f, sum = 0.0f, mine = 0.0f;
    for (int k = 0; k < top; k++) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = z[e];
            if (v > best || (v == best && e < arg)) {
                bool taken = false;
                for (int j = 0; j < k; j++) taken |= picked[j] == e;
                if (!taken) { best = v; arg = e; }
            }
        }
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        if (arg == 0x7fffffff) arg = 0;                 // logits that are not numbers: stay inside the tables
        if (k == 0) zmax = best;
        const float p = expf(best - zmax);
        sum += p;
        if (lane == k) mine = p;
        if (lane == 0) picked[k] = arg;
        __syncwarp();
    }
    if (lane < top) {
        ids[(size_t)t * top + lane] = picked[lane];
        wts[(size_t)t * top + lane] = mine / sum;
    }
}

// A block TB tokens (a row of the router is read once for all of them); a warp a logit, then a warp a token.  all = experts + identities.
template <typename T, int TB>
__global__ void __launch_bounds__(TB == 1 ? 1024 : 256) experts_route_scored_kernel(const T* __restrict__ x, int width, const float* __restrict__ wr,
                                                                   const float* __restrict__ correction, int all, int top, int count, int keep, float scale,
                                                                   int32_t* __restrict__ ids, float* __restrict__ wts, int tokens, int vec, int sigmoid,
                                                                   int squared) {
    extern __shared__ float rs_sm[];                    // [TB][all] scores | [TB][all] choice scores | [TB][count] the groups' best
    dependency_wait();
    let_dependents_start();
    const int t0 = blockIdx.x * TB, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (int e = warp; e < all; e += nwarps) {
        const float* w = wr + (size_t)e * width;
        float acc[TB];
#pragma unroll
        for (int b = 0; b < TB; b++) acc[b] = 0.0f;
        if (vec) {
            constexpr int V = Vec16<T>::N;
#pragma unroll 4
            for (int i = lane * V; i < width; i += 32 * V) {
                float wv[V];
#pragma unroll
                for (int v = 0; v < V; v += 4) *reinterpret_cast<float4*>(wv + v) = *reinterpret_cast<const float4*>(w + i + v);
#pragma unroll
                for (int b = 0; b < TB; b++) {
                    float xv[V];
                    load16<T>(x + (size_t)min(t0 + b, tokens - 1) * width + i, xv);
#pragma unroll
                    for (int v = 0; v < V; v++) acc[b] = fmaf(xv[v], wv[v], acc[b]);
                }
            }
        } else {
            for (int i = lane; i < width; i += 32) {
                const float wv = w[i];
#pragma unroll
                for (int b = 0; b < TB; b++) acc[b] = fmaf(to_f32<T>(x[(size_t)min(t0 + b, tokens - 1) * width + i]), wv, acc[b]);
            }
        }
#pragma unroll
        for (int b = 0; b < TB; b++) {
            acc[b] = warp_sum(acc[b]);
            if (lane == 0) rs_sm[b * all + e] = acc[b];
        }
    }
    __syncthreads();
    const int t = t0 + warp;
    if (warp >= TB || t >= tokens) return;
    float* s = rs_sm + warp * all;
    float* choice = rs_sm + TB * all + warp * all;
    float* best_of = rs_sm + 2 * TB * all + warp * count;
    if (sigmoid) {
        for (int e = lane; e < all; e += 32) {
            const float z = s[e], v = 1.0f / (1.0f + expf(-z));
            s[e] = v;
            choice[e] = correction ? v + correction[e] : z;
        }
    } else {
        float mx = -INFINITY, sum = 0.0f;
        for (int e = lane; e < all; e += 32) mx = fmaxf(mx, s[e]);
        mx = warp_max(mx);
        for (int e = lane; e < all; e += 32) { const float v = expf(s[e] - mx); s[e] = v; sum += v; }
        sum = warp_sum(sum);
        for (int e = lane; e < all; e += 32) {
            const float v = s[e] / sum;
            s[e] = v;
            choice[e] = v + (correction ? correction[e] : 0.0f);
        }
    }
    __syncwarp();
    // the largest of n values (of equals the first), which then counts no more; every lane gets its index
    auto take = [&](float* v, int n) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int i = lane; i < n; i += 32)
            if (v[i] > best) { best = v[i]; arg = i; }
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        if (arg >= n) arg = 0;                          // scores that are not numbers: stay inside the tables
        if (lane == 0) v[arg] = -INFINITY;
        __syncwarp();
        return arg;
    };
    if (keep < count) {
        const int size = all / count;
        for (int g = lane; g < count; g += 32) {
            float m = -INFINITY;
            for (int i = 0; i < size; i++) m = fmaxf(m, choice[g * size + i]);
            best_of[g] = m;
        }
        __syncwarp();
        for (int k = 0; k < keep; k++) take(best_of, count);
        for (int e = lane; e < all; e += 32)
            if (best_of[e / size] != -INFINITY) choice[e] = -INFINITY;      // a group that was not taken
        __syncwarp();
    }
    float mine = 0.0f, chosen = 0.0f;
    int id = 0;
    for (int k = 0; k < top; k++) {
        const int e = take(choice, all);
        chosen += s[e];
        if (lane == k) { mine = s[e]; id = e; }
    }
    if (lane < top) {
        ids[(size_t)t * top + lane] = id;
        const float w = sigmoid ? mine * scale : mine / (chosen + 1e-20f) * scale;
        wts[(size_t)t * top + lane] = squared ? w * w : w;
    }
}

__global__ void __launch_bounds__(256) experts_route_table_kernel(const int32_t* __restrict__ tokens, const int32_t* __restrict__ table, int vocab,
                                                                  int table_top, int E, int top, int32_t* __restrict__ ids, float* __restrict__ wts, int n) {
    dependency_wait();
    let_dependents_start();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int t = i / top, k = i - t * top;
    int id = tokens[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    int e = table[(size_t)id * table_top + k];
    ids[i] = e < 0 ? 0 : (e >= E ? E - 1 : e);         // a table that names no expert of the layer: stay inside the weights
    wts[i] = 1.0f / (float)top;
}

// grid (pairs, column groups); a warp a column.  wgu [E][2 ff][width] (a group's gate rows, then its up rows), or [E][ff][width] ungated
template <typename T, bool GATED>
__global__ void __launch_bounds__(256) experts_gate_up_kernel(const T* __restrict__ x, int width, const T* __restrict__ wgu, int ff, int top,
                                                              const int32_t* __restrict__ ids, int E, int act, float limit, float alpha,
                                                              T* __restrict__ out, int vec) {
    extern __shared__ __align__(16) float xs[];         // [width]
    dependency_wait();
    let_dependents_start();
    const int p = blockIdx.x, t = p / top;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int e = ids[p];
    if (e >= E) return;                                 // an identity
    for (int i = threadIdx.x; i < width; i += blockDim.x) xs[i] = to_f32<T>(x[(size_t)t * width + i]);
    __syncthreads();
    const T* wg = wgu + (size_t)e * (GATED ? 2 : 1) * ff * width;
    const T* wu = wg + (size_t)ff * width;
    for (int c = blockIdx.y * nwarps + warp; c < ff; c += gridDim.y * nwarps) {
        const T* g = wg + (size_t)c * width;
        const T* u = wu + (size_t)c * width;
        float ag = 0.0f, au = 0.0f;
        if (vec) {                                      // 16 bytes of both rows a lane and step
            constexpr int V = Vec16<T>::N;
#pragma unroll 4
            for (int i = lane * V; i < width; i += 32 * V) {
                float gv[V], uv[V];
                load16<T>(g + i, gv);
                if (GATED) load16<T>(u + i, uv);
#pragma unroll
                for (int e = 0; e < V; e += 4) {
                    const float4 x4 = *reinterpret_cast<const float4*>(xs + i + e);
                    ag = fmaf(x4.x, gv[e], ag); ag = fmaf(x4.y, gv[e + 1], ag); ag = fmaf(x4.z, gv[e + 2], ag); ag = fmaf(x4.w, gv[e + 3], ag);
                    if (GATED) { au = fmaf(x4.x, uv[e], au); au = fmaf(x4.y, uv[e + 1], au); au = fmaf(x4.z, uv[e + 2], au); au = fmaf(x4.w, uv[e + 3], au); }
                }
            }
        } else {
            for (int i = lane; i < width; i += 32) {
                ag = fmaf(xs[i], to_f32<T>(g[i]), ag);
                if (GATED) au = fmaf(xs[i], to_f32<T>(u[i]), au);
            }
        }
        ag = warp_sum(ag);
        if (GATED) au = warp_sum(au);
        if (lane == 0) {
            float r;
            if (!GATED) {
                r = activate_dense(act, ag);
            } else if (act == 4) {                             // the clamped form: min(g, L) sigmoid(alpha min(g, L)) (clamp(u, -L, L) + 1)
                const float g = fminf(ag, limit), u = fminf(fmaxf(au, -limit), limit);
                r = (g / (1.0f + expf(-alpha * g))) * (u + 1.0f);
            } else {
                r = activate_rt(act, ag) * au;
            }
            out[(size_t)p * ff + c] = from_f32<T>(r);
        }
    }
}

// grid (tokens, column groups); a warp a column of y
template <typename T>
__global__ void __launch_bounds__(256) experts_down_kernel(const T* __restrict__ act, int ff, const T* __restrict__ wd, int width, int top,
                                                           const int32_t* __restrict__ ids, const float* __restrict__ wts, float* __restrict__ y, int E,
                                                           const T* __restrict__ x, int vec) {
    extern __shared__ __align__(16) float as[];         // [top][ff]
    dependency_wait();
    let_dependents_start();
    const int t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (int i = threadIdx.x; i < top * ff; i += blockDim.x) as[i] = to_f32<T>(act[(size_t)t * top * ff + i]);
    __syncthreads();
    for (int c = blockIdx.y * nwarps + warp; c < width; c += gridDim.y * nwarps) {
        float total = 0.0f;
        for (int k = 0; k < top; k++) {
            const int e = ids[(size_t)t * top + k];
            if (e >= E) {                               // an identity: the input itself
                total = fmaf(wts[(size_t)t * top + k], to_f32<T>(x[(size_t)t * width + c]), total);
                continue;
            }
            const T* w = wd + ((size_t)e * width + c) * ff;
            const float* a = as + (size_t)k * ff;
            float acc = 0.0f;
            if (vec) {
                constexpr int V = Vec16<T>::N;
#pragma unroll 4
                for (int i = lane * V; i < ff; i += 32 * V) {
                    float wv[V];
                    load16<T>(w + i, wv);
#pragma unroll
                    for (int e = 0; e < V; e += 4) {
                        const float4 a4 = *reinterpret_cast<const float4*>(a + i + e);
                        acc = fmaf(a4.x, wv[e], acc); acc = fmaf(a4.y, wv[e + 1], acc); acc = fmaf(a4.z, wv[e + 2], acc); acc = fmaf(a4.w, wv[e + 3], acc);
                    }
                }
            } else {
                for (int i = lane; i < ff; i += 32) acc = fmaf(a[i], to_f32<T>(w[i]), acc);
            }
            total = fmaf(wts[(size_t)t * top + k], warp_sum(acc), total);
        }
        if (lane == 0) y[(size_t)t * width + c] += total;
    }
}

constexpr int ES_PAIRS = 4, ES_STREAMS = 4, ES_MAX_PAIRS = 256;        // pairs a pass; weight rows a warp reads side by side; pairs a step
enum { ES_UP = 0, ES_GATED = 1, ES_DOWN = 2 };

template <typename T, int NP>
__device__ __forceinline__ void es_dots(const T* const* w, const T* rows, int n, int lane, float (*acc)[ES_STREAMS]) {
    constexpr int V = Vec16<T>::N;
#pragma unroll
    for (int p = 0; p < NP; p++)
#pragma unroll
        for (int s = 0; s < ES_STREAMS; s++) acc[p][s] = 0.0f;
#pragma unroll 2
    for (int i = lane * V; i < n; i += 32 * V) {
        float f[ES_STREAMS][V];
#pragma unroll
        for (int s = 0; s < ES_STREAMS; s++) load16<T>(w[s] + i, f[s]);
#pragma unroll
        for (int p = 0; p < NP; p++) {
            float v[V];
            load16<T>(rows + (size_t)p * n + i, v);
#pragma unroll
            for (int s = 0; s < ES_STREAMS; s++)
#pragma unroll
                for (int e = 0; e < V; e++) acc[p][s] = fmaf(v[e], f[s][e], acc[p][s]);
        }
    }
#pragma unroll
    for (int p = 0; p < NP; p++)
#pragma unroll
        for (int s = 0; s < ES_STREAMS; s++) acc[p][s] = warp_sum(acc[p][s]);
}

// grid (E, column groups).  n: the length of a row of the weights and of the inputs; cols: output columns.  ES_GATED, ES_UP: in is x [tokens][n], out
// [pairs][cols] in T; ES_DOWN: in is act [pairs][n], out o float32 [pairs][cols], or (direct) y float32 [tokens][cols], which is added to.
template <typename T, int MODE>
__global__ void __launch_bounds__(256) experts_shared_kernel(const T* __restrict__ in, int n, const T* __restrict__ w, int cols, int top,
                                                             const int32_t* __restrict__ ids, int pairs, int act, float limit, float alpha,
                                                             const float* __restrict__ wts, void* __restrict__ out, int direct) {
    extern __shared__ __align__(16) unsigned char es_sm[];
    T* rows = reinterpret_cast<T*>(es_sm);              // [ES_PAIRS][n]
    __shared__ int list[ES_MAX_PAIRS], counts[8];
    dependency_wait();
    let_dependents_start();
    const int e = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool mine = tid < pairs && ids[tid] == e;
    const unsigned votes = __ballot_sync(0xffffffffu, mine);
    if (lane == 0) counts[warp] = __popc(votes);
    __syncthreads();
    int before = 0, total = 0;
#pragma unroll
    for (int i = 0; i < 8; i++) { before += i < warp ? counts[i] : 0; total += counts[i]; }
    if (total == 0) return;                             // the same for the whole block
    if (mine) list[before + __popc(votes & ((1u << lane) - 1))] = tid;
    constexpr int V = Vec16<T>::N, COLS = MODE == ES_GATED ? ES_STREAMS / 2 : ES_STREAMS;
    const int c0 = (blockIdx.y * 8 + warp) * COLS;
    const T* we = w + (size_t)e * cols * n * (MODE == ES_GATED ? 2 : 1);
    const T* ws[ES_STREAMS];
#pragma unroll
    for (int s = 0; s < ES_STREAMS; s++) {
        const int c = min(c0 + s % COLS, cols - 1);     // a column past the end: read, not written
        ws[s] = we + ((size_t)c + (s >= COLS ? cols : 0)) * n;
    }
    for (int p0 = 0; p0 < total; p0 += ES_PAIRS) {
        const int np = min(ES_PAIRS, total - p0);
        __syncthreads();
        for (int i = tid * V; i < np * n; i += 256 * V) {
            const int p = i / n, d = i - p * n, pair = list[p0 + p];
            *reinterpret_cast<uint4*>(rows + i) = *reinterpret_cast<const uint4*>(in + (size_t)(MODE == ES_DOWN ? pair : pair / top) * n + d);
        }
        __syncthreads();
        if (c0 >= cols) continue;
        float acc[ES_PAIRS][ES_STREAMS];
        if (np == 1) es_dots<T, 1>(ws, rows, n, lane, acc);
        else if (np == 2) es_dots<T, 2>(ws, rows, n, lane, acc);
        else if (np == 3) es_dots<T, 3>(ws, rows, n, lane, acc);
        else es_dots<T, 4>(ws, rows, n, lane, acc);
#pragma unroll
        for (int p = 0; p < ES_PAIRS; p++) {
            if (p >= np) break;
            const int pair = list[p0 + p];
#pragma unroll
            for (int s = 0; s < COLS; s++) {
                const int c = c0 + s;
                if (lane != p * COLS + s || c >= cols) continue;        // every lane has every sum: the lanes share the epilogue out
                if (MODE == ES_DOWN) {
                    if (direct) {
                        float* y = reinterpret_cast<float*>(out) + (size_t)pair * cols + c;
                        *y = __fadd_rn(*y, __fmul_rn(wts[pair], acc[p][s]));     // rounded as the other forms round it
                    }
                    else reinterpret_cast<float*>(out)[(size_t)pair * cols + c] = acc[p][s];
                } else {
                    float r;
                    if (MODE == ES_UP) {
                        r = activate_dense(act, acc[p][s]);
                    } else if (act == 4) {
                        const float g = fminf(acc[p][s], limit), u = fminf(fmaxf(acc[p][s + COLS], -limit), limit);
                        r = (g / (1.0f + expf(-alpha * g))) * (u + 1.0f);
                    } else {
                        r = activate_rt(act, acc[p][s]) * acc[p][s + COLS];
                    }
                    reinterpret_cast<T*>(out)[(size_t)pair * cols + c] = from_f32<T>(r);
                }
            }
        }
    }
}

constexpr int EXPERT_TILE = 128;                        // rows of a tile of the grouped products

__global__ void __launch_bounds__(1024) experts_sort_kernel(const int32_t* __restrict__ ids, int n, int E, int rows_max, int32_t* __restrict__ pos,
                                                            int32_t* __restrict__ row_token, int32_t* __restrict__ tile_group, int top) {
    extern __shared__ int sort_sh[];                    // count [E] | start [E]
    int* count = sort_sh;
    int* start = sort_sh + E;
    dependency_wait();
    let_dependents_start();
    for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
    for (int i = threadIdx.x; i < rows_max; i += blockDim.x) row_token[i] = -1;
    for (int i = threadIdx.x; i < rows_max / EXPERT_TILE; i += blockDim.x) tile_group[i] = -1;
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const int e = ids[i];
        if (e >= 0 && e < E) atomicAdd(&count[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int at = 0;
        for (int e = 0; e < E; e++) {
            start[e] = at;
            at += (count[e] + EXPERT_TILE - 1) / EXPERT_TILE * EXPERT_TILE;
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        for (int r = start[e]; r < start[e] + count[e] && r < rows_max; r += EXPERT_TILE) tile_group[r / EXPERT_TILE] = e;
        count[e] = 0;                                   // from here on: the rows of the group that are taken
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const int e = ids[i];
        int r = -1;
        if (e >= 0 && e < E) {
            r = start[e] + atomicAdd(&count[e], 1);
            if (r < rows_max) row_token[r] = i / top; else r = -1;
        }
        pos[i] = r;
    }
}

template <typename T>
__global__ void __launch_bounds__(128) experts_gather_kernel(const T* __restrict__ x, int width, const int32_t* __restrict__ row_token,
                                                             T* __restrict__ xs) {
    dependency_wait();
    let_dependents_start();
    const int t = row_token[blockIdx.x];
    if (t < 0) return;
    const T* src = x + (size_t)t * width;
    T* dst = xs + (size_t)blockIdx.x * width;
    constexpr int V = Vec16<T>::N;
    if (width % V == 0 && ((uintptr_t)x % 16 == 0) && ((uintptr_t)xs % 16 == 0)) {
        for (int i = threadIdx.x; i < width / V; i += blockDim.x) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
    } else {
        for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
    }
}

template <typename T>
__global__ void __launch_bounds__(256) experts_combine_kernel(const float* __restrict__ o, int width, int top, const int32_t* __restrict__ pos,
                                                              const float* __restrict__ wts, float* __restrict__ y, int E,
                                                              const int32_t* __restrict__ ids, const T* __restrict__ x) {
    dependency_wait();
    let_dependents_start();
    const int t = blockIdx.x;
    if (width % 4 == 0 && ((uintptr_t)o % 16) == 0 && ((uintptr_t)y % 16) == 0 && ((uintptr_t)x % 16) == 0) {
        for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
            float4 sum = *reinterpret_cast<const float4*>(y + (size_t)t * width + c);
            float4 total = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            for (int k = 0; k < top; k++) {
                const int r = pos ? pos[(size_t)t * top + k] : (ids[(size_t)t * top + k] < E ? t * top + k : -1);
                const float w = wts[(size_t)t * top + k];
                float4 v;
                if (r >= 0) {
                    v = *reinterpret_cast<const float4*>(o + (size_t)r * width + c);
                } else if (ids[(size_t)t * top + k] >= E) {
                    const T* p = x + (size_t)t * width + c;
                    v = make_float4(to_f32<T>(p[0]), to_f32<T>(p[1]), to_f32<T>(p[2]), to_f32<T>(p[3]));
                } else {
                    continue;
                }
                total.x = fmaf(w, v.x, total.x); total.y = fmaf(w, v.y, total.y); total.z = fmaf(w, v.z, total.z); total.w = fmaf(w, v.w, total.w);
            }
            sum.x += total.x; sum.y += total.y; sum.z += total.z; sum.w += total.w;
            *reinterpret_cast<float4*>(y + (size_t)t * width + c) = sum;
        }
        return;
    }
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float total = 0.0f;
        for (int k = 0; k < top; k++) {
            const int r = pos ? pos[(size_t)t * top + k] : (ids[(size_t)t * top + k] < E ? t * top + k : -1);
            if (r >= 0) total = fmaf(wts[(size_t)t * top + k], o[(size_t)r * width + c], total);
            else if (ids[(size_t)t * top + k] >= E) total = fmaf(wts[(size_t)t * top + k], to_f32<T>(x[(size_t)t * width + c]), total);
        }
        y[(size_t)t * width + c] += total;
    }
}

}  // namespace vk

using namespace vk;

// Rows that the grouped matrix needs for `tokens` tokens at most: every copy, and every group filled up to a whole tile.
VK_API int vk_experts_grouped_rows(int tokens, int top, int E) {
    const long long rows = ((long long)tokens * top + (long long)E * (EXPERT_TILE - 1) + EXPERT_TILE - 1) / EXPERT_TILE * EXPERT_TILE;
    return rows > 0x7fffffffLL ? -1 : (int)rows;
}

// ids int32 [tokens][top] -> pos int32 [tokens][top], row_token int32 [rows_max], tile_group int32 [rows_max / 128];
// rows_max = vk_experts_grouped_rows(tokens, top, E).
VK_API int vk_experts_sort(const int32_t* ids, int tokens, int top, int E, int rows_max, int32_t* pos, int32_t* row_token, int32_t* tile_group,
                           cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (top <= 0 || E <= 0 || rows_max < vk_experts_grouped_rows(tokens, top, E) || rows_max % EXPERT_TILE) return VK_BAD_SHAPE;
    const size_t smem = 2 * (size_t)E * sizeof(int);
    if (smem > 48 * 1024) return VK_TOO_LARGE;
    return launch_dependent(experts_sort_kernel, dim3(1), dim3(1024), smem, stream, ids, tokens * top, E, rows_max, pos, row_token, tile_group, top);
}

// xs [rows][width] in dtype <- x [tokens][width] by row_token.
VK_API int vk_experts_gather(const void* x, int width, const int32_t* row_token, void* xs, int rows, int dtype, cudaStream_t stream) {
    if (rows <= 0) return VK_OK;
    if (width <= 0) return VK_BAD_SHAPE;
    if (dtype == 0) return launch_dependent(experts_gather_kernel<float>, dim3(rows), dim3(128), 0, stream, (const float*)x, width, row_token, (float*)xs);
    return launch_dependent(experts_gather_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, stream, (const __nv_bfloat16*)x, width, row_token,
                            (__nv_bfloat16*)xs);
}

// pos null: a token's rows of o are t * top + k.  y float32 [tokens][width] += sum_k wts[t][k] o[pos[t][k]]; o float32 [rows][width]; ids of E and more: the token's row of x [tokens][width].
VK_API int vk_experts_combine(const float* o, int width, int top, const int32_t* pos, const float* wts, float* y, int E, const int32_t* ids, const void* x,
                              int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || top <= 0) return VK_BAD_SHAPE;
    if (dtype == 0)
        return launch_dependent(experts_combine_kernel<float>, dim3(tokens), dim3(256), 0, stream, o, width, top, pos, wts, y, E, ids, (const float*)x);
    return launch_dependent(experts_combine_kernel<__nv_bfloat16>, dim3(tokens), dim3(256), 0, stream, o, width, top, pos, wts, y, E, ids,
                            (const __nv_bfloat16*)x);
}

// x [tokens][width] in dtype; wr float32 [all][width], correction float32 [all] or null, all = experts + identities, in `count` equal groups of
// neighbours of which `keep` take part; ids int32 [tokens][top], wts float32 [tokens][top].  sigmoid 1: the form with a sigmoid a score;
// squared 1: the weights' squares.
VK_API int vk_experts_route_scored(const void* x, int width, const float* wr, const float* correction, int all, int top, int count, int keep, float scale,
                                   int sigmoid, int squared, int32_t* ids, float* wts, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || all <= 0 || count <= 0 || all % count || keep <= 0 || keep > count || top <= 0 || top > 32 || top > all / count * keep) return VK_BAD_SHAPE;
    const int tb = tokens > 64 ? 4 : 1;
    const size_t smem = (size_t)tb * (2 * all + count) * sizeof(float);
    if (smem > 48 * 1024) return VK_TOO_LARGE;
    const dim3 grid((tokens + tb - 1) / tb);
    const int vec = width % (dtype == 0 ? 4 : 8) == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)wr % 16) == 0;
    int warps = tb == 1 && all > 8 ? all : 8;           // few tokens: a warp a logit, as far as a block has warps
    if (warps > 32) warps = 32;
#define VK_ERS(T, TB)                                                                                                                          \
    return launch_dependent(experts_route_scored_kernel<T, TB>, grid, dim3(32 * warps), smem, stream, (const T*)x, width, wr, correction, all, top, count, \
                            keep, scale, ids, wts, tokens, vec, sigmoid, squared)
    if (dtype == 0) {
        if (tb == 4) VK_ERS(float, 4);
        VK_ERS(float, 1);
    }
    if (tb == 4) VK_ERS(__nv_bfloat16, 4);
    VK_ERS(__nv_bfloat16, 1);
#undef VK_ERS
}

// x [tokens][width] in dtype; wr float32 [E][width], br float32 [E] or null; ids int32 [tokens][top], wts float32 [tokens][top].
VK_API int vk_experts_route(const void* x, int width, const float* wr, const float* br, int E, int top, int32_t* ids, float* wts, int tokens,
                            int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || E <= 0 || top <= 0 || top > E || top > 32) return VK_BAD_SHAPE;
    const size_t smem = (size_t)E * sizeof(float);
    if (smem > 48 * 1024) return VK_TOO_LARGE;
    if (dtype == 0) return launch_dependent(experts_route_kernel<float>, dim3(tokens), dim3(128), smem, stream, (const float*)x, width, wr, br, E, top, ids, wts);
    return launch_dependent(experts_route_kernel<__nv_bfloat16>, dim3(tokens), dim3(128), smem, stream, (const __nv_bfloat16*)x, width, wr, br, E, top,
                            ids, wts);
}

// Whether the kernels for tokens that share experts take these sizes (the launchers below refuse the others).
VK_API int vk_experts_shared_takes(int pairs, int width, int ff, int dtype) {
    const int v = dtype == 0 ? 4 : 8, size = dtype == 0 ? 4 : 2, longest = width > ff ? width : ff;
    return pairs > 0 && pairs <= ES_MAX_PAIRS && width % v == 0 && ff % v == 0 && (size_t)ES_PAIRS * longest * size <= 200 * 1024;
}

template <typename T, int MODE>
static int launch_shared(const void* in, int n, const void* w, int cols, int top, const int32_t* ids, int pairs, int E, int act, float limit, float alpha,
                         const float* wts, void* out, int direct, cudaStream_t stream) {
    auto kern = experts_shared_kernel<T, MODE>;
    const size_t smem = (size_t)ES_PAIRS * n * sizeof(T);
    if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    constexpr int COLS = 8 * (MODE == ES_GATED ? ES_STREAMS / 2 : ES_STREAMS);
    const dim3 grid(E, (cols + COLS - 1) / COLS);
    if (grid.y > 65535) return VK_TOO_LARGE;
    return launch_dependent(kern, grid, dim3(256), smem, stream, (const T*)in, n, (const T*)w, cols, top, ids, pairs, act, limit, alpha, wts, out, direct);
}

// vk_experts_gate_up for up to 256 (token, k) pairs.
VK_API int vk_experts_shared_up(const void* x, int width, const void* wgu, int ff, int top, const int32_t* ids, int E, int gated, int act, float limit,
                                float alpha, void* out, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || ff <= 0 || top <= 0 || E <= 0 || act < 0 || act > 4 || (gated && act == 4 && !(limit > 0.0f))) return VK_BAD_SHAPE;
    if (!vk_experts_shared_takes(tokens * top, width, ff, dtype)) return VK_BAD_SHAPE;
    if (((uintptr_t)x % 16) || ((uintptr_t)wgu % 16)) return VK_BAD_ALIGNMENT;
    const int pairs = tokens * top;
#define VK_ES(T, MODE) return launch_shared<T, MODE>(x, width, wgu, ff, top, ids, pairs, E, act, limit, alpha, nullptr, out, 0, stream)
    if (dtype == 0) { if (gated) VK_ES(float, ES_GATED); VK_ES(float, ES_UP); }
    if (gated) VK_ES(__nv_bfloat16, ES_GATED);
    VK_ES(__nv_bfloat16, ES_UP);
#undef VK_ES
}

// act [tokens * top][ff] and wd [E][width][ff] in dtype.  direct 0: out float32 [tokens * top][width], a row a pair (vk_experts_combine follows);
// direct 1 (top 1, no identities): out is y float32 [tokens][width], and wts[t] times the row is added to it.
VK_API int vk_experts_shared_down(const void* act, int ff, const void* wd, int width, int top, const int32_t* ids, const float* wts, float* out, int E,
                                  int direct, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || ff <= 0 || top <= 0 || E <= 0 || (direct && top != 1)) return VK_BAD_SHAPE;
    if (!vk_experts_shared_takes(tokens * top, width, ff, dtype)) return VK_BAD_SHAPE;
    if (((uintptr_t)act % 16) || ((uintptr_t)wd % 16)) return VK_BAD_ALIGNMENT;
    const int pairs = tokens * top;
    if (dtype == 0) return launch_shared<float, ES_DOWN>(act, ff, wd, width, top, ids, pairs, E, 0, 0.0f, 0.0f, wts, out, direct, stream);
    return launch_shared<__nv_bfloat16, ES_DOWN>(act, ff, wd, width, top, ids, pairs, E, 0, 0.0f, 0.0f, wts, out, direct, stream);
}

// tokens int32 [n_tokens] (token ids); table int32 [vocab][table_top], table_top >= top; ids int32 [n_tokens][top], wts float32 [n_tokens][top].
VK_API int vk_experts_route_table(const int32_t* tokens, const int32_t* table, int vocab, int table_top, int E, int top, int32_t* ids, float* wts,
                                  int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return VK_OK;
    if (vocab <= 0 || E <= 0 || top <= 0 || top > table_top) return VK_BAD_SHAPE;
    const int n = n_tokens * top;
    return launch_dependent(experts_route_table_kernel, dim3((n + 255) / 256), dim3(256), 0, stream, tokens, table, vocab, table_top, E, top, ids, wts, n);
}

// wgu [E][2 ff][width] (an expert's gate rows, then its up rows) in dtype; out [tokens * top][ff] in dtype.  act: 0 none, 1 gelu (erf),
// 2 gelu (tanh), 3 silu, 4 the clamped form min(g, limit) sigmoid(alpha min(g, limit)) (clamp(u, -limit, limit) + 1).
// gated 0: wgu [E][ff][width], and act as activate_dense numbers them (4 is relu squared).
VK_API int vk_experts_gate_up(const void* x, int width, const void* wgu, int ff, int top, const int32_t* ids, int E, int gated, int act, float limit,
                              float alpha, void* out, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || ff <= 0 || top <= 0 || act < 0 || act > 4 || (gated && act == 4 && !(limit > 0.0f))) return VK_BAD_SHAPE;
    const size_t smem = (size_t)width * sizeof(float);
    if (smem > 48 * 1024) return VK_TOO_LARGE;
    int gy = (ff + 7) / 8;
    if (gy > 64) gy = 64;
    dim3 grid(tokens * top, gy);
    const int vec = width % (dtype == 0 ? 4 : 8) == 0 && ((uintptr_t)wgu % 16) == 0;
    auto go = [&](auto kf, auto kb) {
        if (dtype == 0)
            return launch_dependent(kf, grid, dim3(256), smem, stream, (const float*)x, width, (const float*)wgu, ff, top, ids, E, act, limit, alpha,
                                    (float*)out, vec);
        return launch_dependent(kb, grid, dim3(256), smem, stream, (const __nv_bfloat16*)x, width, (const __nv_bfloat16*)wgu, ff, top, ids, E, act, limit,
                                alpha, (__nv_bfloat16*)out, vec);
    };
    if (gated) return go(experts_gate_up_kernel<float, true>, experts_gate_up_kernel<__nv_bfloat16, true>);
    return go(experts_gate_up_kernel<float, false>, experts_gate_up_kernel<__nv_bfloat16, false>);
}

// act [tokens * top][ff] and wd [E][width][ff] in dtype; y float32 [tokens][width] is added to; ids of E and more: the token's row of x.
VK_API int vk_experts_down(const void* act, int ff, const void* wd, int width, int top, const int32_t* ids, const float* wts, float* y, int E,
                           const void* x, int tokens, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VK_OK;
    if (width <= 0 || ff <= 0 || top <= 0) return VK_BAD_SHAPE;
    const size_t smem = (size_t)top * ff * sizeof(float);
    if (smem > 200 * 1024) return VK_TOO_LARGE;
    int gy = (width + 7) / 8;
    if (gy > 64) gy = 64;
    dim3 grid(tokens, gy);
    const int vec = ff % (dtype == 0 ? 4 : 8) == 0 && ((uintptr_t)wd % 16) == 0;
    if (smem > 48 * 1024) {
        cudaError_t e = dtype == 0 ? cudaFuncSetAttribute(experts_down_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
                                   : cudaFuncSetAttribute(experts_down_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    if (dtype == 0)
        return launch_dependent(experts_down_kernel<float>, grid, dim3(256), smem, stream, (const float*)act, ff, (const float*)wd, width, top, ids, wts, y,
                                E, (const float*)x, vec);
    return launch_dependent(experts_down_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, (const __nv_bfloat16*)act, ff, (const __nv_bfloat16*)wd,
                            width, top, ids, wts, y, E, (const __nv_bfloat16*)x, vec);
}
