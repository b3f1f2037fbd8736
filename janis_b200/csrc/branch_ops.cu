// Rows of the residual stream and of a layer's branches: the sum that a sublayer's result joins with the norm behind it, the Dynamic Tanh norm, the RMS norm in groups that follows a
// scaled residual sum, the norm-and-accumulate of branches that run side by side, and a sigmoid gate on the heads of
// an attention.  All arithmetic is float.
#include "common.cuh"

#include <math_constants.h>

namespace janis {

// h[r] += res[r] (when res is given: the float residual sum, in place), then
// y[r] = tanh(alpha * h[src]) * w + b with src = rows[r] (or r): no statistics of the row are taken.
template <typename TR, typename TO>
__global__ void __launch_bounds__(256)
dyt_norm_kernel(float* __restrict__ h, const TR* __restrict__ res, const int* __restrict__ rows, float alpha,
                const float* __restrict__ w, const float* __restrict__ b, TO* __restrict__ y, int H) {
    const int r = blockIdx.x;
    grid_dependents_launch();
    grid_dependency_wait();
    const int src = rows != nullptr ? rows[r] : r;
    float* hr = h + (size_t)src * H;
    TO* yr = y + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float v = hr[i];
        if (res != nullptr) {
            v += to_float(res[(size_t)r * H + i]);
            hr[i] = v;
        }
        yr[i] = from_float<TO>(fmaf(tanhf(alpha * v), w[i], b[i]));
    }
}

// acc[r] = (first ? 0 : acc[r]) + share * x[r] / sqrt(mean(x[r]^2) + eps) * w
template <typename T>
__global__ void __launch_bounds__(256)
rmsnorm_accumulate_kernel(const T* __restrict__ x, const float* __restrict__ w, float eps, float share,
                          float* __restrict__ acc, int first, int H) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    grid_dependents_launch();
    grid_dependency_wait();
    const T* xr = x + (size_t)r * H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_float(xr[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = share / sqrtf(ss / (float)H + eps);
    float* ar = acc + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_float(xr[i]) * inv * w[i];
        ar[i] = first ? v : ar[i] + v;
    }
}

// RMS norm in groups: the row is cut into `groups` equal runs, each divided by sqrt(mean(run^2) + eps), and the whole
// multiplied by w.  With a residual: v = alpha h[r] + res[r], h[r] = norm(v) (the stream itself is normed, in place)
// and y[r] = h[r] rounded; without: y[r] = norm(h[src]) with src = rows[r] (or r), h untouched.
// A group's sum runs over the lanes of its warps and then over its warps in index order.
__device__ __forceinline__ void load4(const float* p, float* o) { Vec16<float>::load(p, o); }
__device__ __forceinline__ void load4(const bf16* p, float* o) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xffff0000u);
    o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float* v) { Vec16<float>::store(p, v); }
__device__ __forceinline__ void store4(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

// VEC: four elements a load and a store (a group's length is a multiple of four, and so is every row's start)
template <typename TR, typename TO, bool VEC>
__global__ void __launch_bounds__(256)
group_norm_kernel(float* __restrict__ h, const TR* __restrict__ res, const int* __restrict__ rows, float alpha,
                  const float* __restrict__ w, float eps, int groups, TO* __restrict__ y, int H) {
    extern __shared__ float gn_smem[];
    float* row_s = gn_smem;                 // the row
    float* inv_s = row_s + H;               // 1 / rms of each group
    float* scratch = inv_s + groups;        // a partial sum per warp
    const int r = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarp = blockDim.x >> 5;
    grid_dependents_launch();
    grid_dependency_wait();
    const int src = rows != nullptr ? rows[r] : r;
    float* hr = h + (size_t)src * H;
    if (VEC) {
        for (int i = tid * 4; i < H; i += blockDim.x * 4) {
            float v[4], a[4];
            load4(hr + i, v);
            if (res != nullptr) {
                load4(res + (size_t)r * H + i, a);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] = fmaf(alpha, v[e], a[e]);
            }
            store4(row_s + i, v);
        }
    } else {
        for (int i = tid; i < H; i += blockDim.x) {
            float v = hr[i];
            if (res != nullptr) v = fmaf(alpha, v, to_float(res[(size_t)r * H + i]));
            row_s[i] = v;
        }
    }
    const int gs = H / groups;
    const int wpg = nwarp / groups > 0 ? nwarp / groups : 1;      // warps that share a group
    const int gpr = nwarp / wpg;                                  // groups summed side by side
    for (int g0 = 0; g0 < groups; g0 += gpr) {
        __syncthreads();
        const int g = g0 + warp / wpg, wi = warp % wpg;
        float ss = 0.f;
        if (g < groups && warp < gpr * wpg)
            for (int i = wi * 32 + lane; i < gs; i += wpg * 32) {
                const float v = row_s[g * gs + i];
                ss = fmaf(v, v, ss);
            }
        ss = warp_sum(ss);
        if (lane == 0) scratch[warp] = ss;
        __syncthreads();
        if (tid < gpr && g0 + tid < groups) {
            float tot = 0.f;
            for (int k = 0; k < wpg; ++k) tot += scratch[tid * wpg + k];
            inv_s[g0 + tid] = 1.f / sqrtf(tot / (float)gs + eps);
        }
    }
    __syncthreads();
    if (VEC) {
        for (int i = tid * 4; i < H; i += blockDim.x * 4) {
            float v[4], ww[4];
            load4(row_s + i, v);
            load4(w + i, ww);
            const float inv = inv_s[i / gs];
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = v[e] * inv * ww[e];
            if (res != nullptr) store4(hr + i, v);
            if (y != nullptr) store4(y + (size_t)r * H + i, v);
        }
    } else {
        for (int i = tid; i < H; i += blockDim.x) {
            const float v = row_s[i] * inv_s[i / gs] * w[i];
            if (res != nullptr) hr[i] = v;
            if (y != nullptr) y[(size_t)r * H + i] = from_float<TO>(v);
        }
    }
}

// ---------------------------------------------------------------------------
// A sublayer's result into the stream, and the norm behind the sum:
//
//   v    = r0                                                  one branch as it is, or
//   v    = share * (rms(r0) * w0 + rms(r1) * w1)               one or two branches normed first (w0, w1 given)
//   h[r] += scale * v + more[r]                                scale: a factor per feature (null: 1); more: rows of the
//                                                              stream's type that join the sum (null: none)
//   y[r] = norm(h[r]) * w_next                                 centred: (h - mean) / sqrt(mean((h - mean)^2) + eps),
//                                                              else h / sqrt(mean(h^2) + eps)
//
// With r0 null nothing is added and y[r] = norm(h[rows[r] or r]), h untouched.
// ---------------------------------------------------------------------------
struct StreamSum {
    const float* w0;          // the branches' norm weights, or null
    const float* w1;
    float eps, share;
    const float* scale;
    const float* more;
};

// two sums over the block at once, in the order of block_sum
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
    for (int w = 0; w < nwarp; ++w) {
        t.x += scratch[w].x;
        t.y += scratch[w].y;
    }
    return t;
}

// VW elements an access: 4 (rows of whole 16-byte pieces; the row stays in registers, up to VPT pieces a thread) or 1 (any
// row; the row is read again from where it was written).
template <typename TR, typename TO, int VW, int VPT>
__global__ void __launch_bounds__(256)
stream_norm_kernel(float* __restrict__ h, const TR* __restrict__ r0, const TR* __restrict__ r1, StreamSum s,
                   const float* __restrict__ w_next, float eps_next, int centred, TO* __restrict__ y,
                   const int* __restrict__ rows, int H) {
    __shared__ float2 scratch2[32];
    __shared__ float scratch[32];
    const int r = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
    grid_dependents_launch();
    grid_dependency_wait();
    float* hr = h + (size_t)(rows != nullptr ? rows[r] : r) * H;
    const TR* a0 = r0 != nullptr ? r0 + (size_t)r * H : nullptr;
    const TR* a1 = r1 != nullptr ? r1 + (size_t)r * H : nullptr;
    const float* mr = s.more != nullptr ? s.more + (size_t)r * H : nullptr;
    const float n = (float)H;
    if (VW == 4) {
        const int pieces = H >> 2;
        float hv[VPT][4];
#pragma unroll
        for (int p = 0; p < VPT; ++p) {
            const int i = (tid + p * nt) * 4;
            hv[p][0] = hv[p][1] = hv[p][2] = hv[p][3] = 0.f;
            if (tid + p * nt < pieces) load4(hr + i, hv[p]);
        }
        float sum = 0.f;
        if (a0 != nullptr) {
            float inv0 = 1.f, inv1 = 0.f;
            float v0[VPT][4], v1[VPT][4];
#pragma unroll
            for (int p = 0; p < VPT; ++p) {
                const int i = (tid + p * nt) * 4;
                const bool in = tid + p * nt < pieces;
#pragma unroll
                for (int e = 0; e < 4; ++e) v0[p][e] = v1[p][e] = 0.f;
                if (in) load4(a0 + i, v0[p]);
                if (in && a1 != nullptr) load4(a1 + i, v1[p]);
            }
            if (s.w0 != nullptr) {
                float s0 = 0.f, s1 = 0.f;
#pragma unroll
                for (int p = 0; p < VPT; ++p)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        s0 = fmaf(v0[p][e], v0[p][e], s0);
                        s1 = fmaf(v1[p][e], v1[p][e], s1);
                    }
                const float2 t = block_sum2(s0, s1, scratch2);
                inv0 = s.share / sqrtf(t.x / n + s.eps);
                inv1 = s.share / sqrtf(t.y / n + s.eps);
            }
#pragma unroll
            for (int p = 0; p < VPT; ++p) {
                const int i = (tid + p * nt) * 4;
                if (tid + p * nt >= pieces) continue;
                float w[4];
                if (s.w0 != nullptr) {
                    load4(s.w0 + i, w);
#pragma unroll
                    for (int e = 0; e < 4; ++e) v0[p][e] *= inv0 * w[e];
                    if (a1 != nullptr) {
                        load4(s.w1 + i, w);
#pragma unroll
                        for (int e = 0; e < 4; ++e) v0[p][e] = fmaf(v1[p][e] * inv1, w[e], v0[p][e]);
                    }
                }
                if (s.scale != nullptr) {
                    load4(s.scale + i, w);
#pragma unroll
                    for (int e = 0; e < 4; ++e) hv[p][e] = fmaf(w[e], v0[p][e], hv[p][e]);
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) hv[p][e] += v0[p][e];
                }
                if (mr != nullptr) {
                    load4(mr + i, w);
#pragma unroll
                    for (int e = 0; e < 4; ++e) hv[p][e] += w[e];
                }
                store4(hr + i, hv[p]);
            }
        }
        if (w_next == nullptr) return;
        float mean = 0.f;
        if (centred) {
#pragma unroll
            for (int p = 0; p < VPT; ++p)
#pragma unroll
                for (int e = 0; e < 4; ++e) sum += hv[p][e];
            mean = block_sum(sum, scratch) / n;
        }
        float ss = 0.f;
#pragma unroll
        for (int p = 0; p < VPT; ++p)
            if (tid + p * nt < pieces) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    hv[p][e] -= mean;
                    ss = fmaf(hv[p][e], hv[p][e], ss);
                }
            }
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / n + eps_next);
#pragma unroll
        for (int p = 0; p < VPT; ++p) {
            const int i = (tid + p * nt) * 4;
            if (tid + p * nt >= pieces) continue;
            float w[4], o[4];
            load4(w_next + i, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] = hv[p][e] * inv * w[e];
            store4(y + (size_t)r * H + i, o);
        }
        return;
    }
    float sum = 0.f;
    if (a0 != nullptr) {
        float inv0 = 1.f, inv1 = 0.f;
        if (s.w0 != nullptr) {
            float s0 = 0.f, s1 = 0.f;
            for (int i = tid; i < H; i += nt) {
                const float u = to_float(a0[i]), v = a1 != nullptr ? to_float(a1[i]) : 0.f;
                s0 = fmaf(u, u, s0);
                s1 = fmaf(v, v, s1);
            }
            const float2 t = block_sum2(s0, s1, scratch2);
            inv0 = s.share / sqrtf(t.x / n + s.eps);
            inv1 = s.share / sqrtf(t.y / n + s.eps);
        }
        for (int i = tid; i < H; i += nt) {
            float v = to_float(a0[i]);
            if (s.w0 != nullptr) {
                v *= inv0 * s.w0[i];
                if (a1 != nullptr) v = fmaf(to_float(a1[i]) * inv1, s.w1[i], v);
            }
            float hv = s.scale != nullptr ? fmaf(s.scale[i], v, hr[i]) : hr[i] + v;
            if (mr != nullptr) hv += mr[i];
            hr[i] = hv;                          // read back below by this same thread only
            sum += hv;
        }
    } else if (centred) {
        for (int i = tid; i < H; i += nt) sum += hr[i];
    }
    if (w_next == nullptr) return;
    const float mean = centred ? block_sum(sum, scratch) / n : 0.f;
    float ss = 0.f;
    for (int i = tid; i < H; i += nt) {
        const float v = hr[i] - mean;
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / n + eps_next);
    for (int i = tid; i < H; i += nt) y[(size_t)r * H + i] = from_float<TO>((hr[i] - mean) * inv * w_next[i]);
}

// y = h rounded to the activation type: what a sublayer reads when it reads the stream itself
__global__ void __launch_bounds__(256) round_rows_kernel(const float* __restrict__ h, bf16* __restrict__ y, size_t n) {
    grid_dependents_launch();
    grid_dependency_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        y[i] = __float2bfloat16_rn(h[i]);
}

// x[t, c] *= sigmoid(rows[t, g_off + c / per]): a gate per element (per = 1) or per run of `per` elements (a head)
template <typename T>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(T* __restrict__ x, const T* __restrict__ rows, int row_elems, int g_off, int width, int per, size_t n) {
    grid_dependents_launch();
    grid_dependency_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / width;
        const int c = (int)(i % width) / per;
        const float g = to_float(rows[t * row_elems + g_off + c]);
        x[i] = from_float<T>(to_float(x[i]) / (1.0f + expf(-g)));
    }
}

// ---------------------------------------------------------------------------
// Mixture of experts: the router and the experts' activation.
//
// router, a warp per token over E logits z (float):  s = sigmoid(z), c = s + correction;  experts form n_groups equal
// groups of neighbours, a group's score is the sum of its two largest c (group_best: its largest), the best `keep` groups stay (ties: the
// lower index); among their experts the `top` of largest c are chosen (ties: the lower index); the chosen get
// w_e = s_e / (sum of the chosen s + 1e-20) * scale (raw: w_e = s_e * scale), every other expert 0.  With a shared gate, column E of z is
// its logit and column E of the output its sigmoid.  With `softmax` the scores are the softmax of z over all entries instead.  With
// n_identity > 0 the router scores that many entries more, behind the experts (no groups then); they have no column of
// their own in the output: the weights of the chosen ones add up in its last column.
// ---------------------------------------------------------------------------
constexpr int ROUTE_WARPS = 4;

__device__ __forceinline__ void warp_argmax(float& v, int& at) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ov > v || (ov == v && oa < at)) { v = ov; at = oa; }
    }
}

__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ z, const float* __restrict__ correction, int T, int E, int n_groups, int keep,
                 int top, float scale, int shared_gate, float* __restrict__ out, int n_identity, int softmax, int group_best, int raw) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * ROUTE_WARPS + warp;
    const int N = E + n_identity;                    // entries the router scores: the experts, then the identity entries
    float* s = smem + (size_t)warp * (4 * N);        // scores
    float* c = s + N;                                // choice scores (minus infinity once out of the running)
    float* gs = c + N;                               // group scores
    float* mark = gs + N;                            // 1 for the chosen
    grid_dependents_launch();
    grid_dependency_wait();
    if (t >= T) return;
    const int cols_in = N + (shared_gate ? 1 : 0), cols_out = E + (shared_gate ? 1 : 0) + (n_identity ? 1 : 0), per = N / n_groups;
    const float* zr = z + (size_t)t * cols_in;
    float* o = out + (size_t)t * cols_out;
    float zmax = -CUDART_INF_F, zsum = 0.f;
    if (softmax) {
        for (int e = lane; e < N; e += 32) zmax = fmaxf(zmax, zr[e]);
        zmax = warp_max(zmax);
        for (int e = lane; e < N; e += 32) {
            const float v = expf(zr[e] - zmax);
            s[e] = v;
            zsum += v;
        }
        zsum = warp_sum(zsum);
    }
    for (int e = lane; e < N; e += 32) {
        const float v = softmax ? s[e] / zsum : 1.0f / (1.0f + expf(-zr[e]));
        s[e] = v;
        c[e] = correction != nullptr ? v + correction[e] : v;
        mark[e] = 0.f;
    }
    if (shared_gate && lane == 0) o[E] = 1.0f / (1.0f + expf(-zr[N]));
    __syncwarp();
    if (n_groups > 1 && keep < n_groups) {
        for (int g = lane; g < n_groups; g += 32) {
            float a = -CUDART_INF_F, b = -CUDART_INF_F;      // the two largest
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = c[e];
                if (v > a) { b = a; a = v; }
                else if (v > b) b = v;
            }
            gs[g] = per > 1 && !group_best ? a + b : a;
        }
        __syncwarp();
        // the kept groups get +inf as a mark; the others' experts leave the running
        for (int k = 0; k < keep; ++k) {
            float v = -CUDART_INF_F;
            int at = 0x7fffffff;
            for (int g = lane; g < n_groups; g += 32) {
                const float gv = gs[g];
                if (gv != CUDART_INF_F && (gv > v || (gv == v && g < at))) { v = gv; at = g; }
            }
            warp_argmax(v, at);
            __syncwarp();
            if (lane == 0 && at < n_groups) gs[at] = CUDART_INF_F;
            __syncwarp();
        }
        for (int e = lane; e < N; e += 32)
            if (gs[e / per] != CUDART_INF_F) c[e] = -CUDART_INF_F;
        __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float v = -CUDART_INF_F;
        int at = 0x7fffffff;
        for (int e = lane; e < N; e += 32) {
            const float cv = c[e];
            if (cv > v || (cv == v && e < at)) { v = cv; at = e; }
        }
        warp_argmax(v, at);
        __syncwarp();
        if (at >= N) break;                          // nothing left in the running
        total += s[at];
        if (lane == 0) {
            c[at] = -CUDART_INF_F;
            mark[at] = 1.f;
        }
        __syncwarp();
    }
    const float f = raw ? scale : scale / (total + 1e-20f);
    for (int e = lane; e < E; e += 32) o[e] = mark[e] != 0.f ? s[e] * f : 0.f;
    if (n_identity) {
        float id = 0.f;                              // the identity entries' weights add up: they all return the input
        for (int e = E + lane; e < N; e += 32)
            if (mark[e] != 0.f) id += s[e] * f;
        id = warp_sum(id);
        if (lane == 0) o[cols_out - 1] = id;
    }
}

// out[t, :] += w[t] y[t, :], w[t] = wts[t, w_col]: what the chosen identity entries of a mixture add to its output
template <typename T>
__global__ void __launch_bounds__(256)
moe_identity_add_kernel(T* __restrict__ out, const T* __restrict__ y, const float* __restrict__ wts, int wts_stride, int w_col,
                        int width, size_t n) {
    grid_dependents_launch();
    grid_dependency_wait();
    constexpr int V = Vec16<T>::N;
    if (width % V == 0 && (((uintptr_t)out | (uintptr_t)y) & 15) == 0) {
        // 16 bytes a thread; the pieces of a row share its weight
        for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V) {
            const float w = wts[(i / width) * wts_stride + w_col];
            if (w == 0.f) continue;
            float a[V], b[V];
            Vec16<T>::load(out + i, a);
            Vec16<T>::load(y + i, b);
#pragma unroll
            for (int e = 0; e < V; ++e) a[e] = fmaf(w, b[e], a[e]);
            Vec16<T>::store(out + i, a);
        }
        return;
    }
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const float w = wts[(i / width) * wts_stride + w_col];
        if (w != 0.f) out[i] = from_float<T>(fmaf(w, to_float(y[i]), to_float(out[i])));
    }
}

// a[t, col] = w[t, e] * g sigmoid(alpha g) (u + up_add), g = min(gate, limit), u = clamp(up, -limit, limit), over the
// columns of all experts side by side (expert e: `ff` columns; then the shared expert's `shared_ff`); in gu an
// expert's gate columns are followed by its up columns.  Experts of weight 0 give exact zeros.  w_in: the weight stands on
// the expert's input instead, so that gate and up (which are linear in it) are multiplied by w and the result is not.
template <typename T>
__global__ void __launch_bounds__(256)
moe_expert_act_kernel(const T* __restrict__ gu, const float* __restrict__ wts, int E, int ff, float limit, int shared_ff,
                      float shared_limit, float alpha, T* __restrict__ out, size_t n, int wcols, float up_add, int w_in) {
    const int total = E * ff + shared_ff;
    grid_dependents_launch();
    grid_dependency_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / total;
        const int col = (int)(i % total);
        int e, j, width;
        float lim;
        size_t base;
        if (col < E * ff) { e = col / ff; j = col % ff; width = ff; lim = limit; base = (size_t)2 * e * ff; }
        else { e = E; j = col - E * ff; width = shared_ff; lim = shared_limit; base = (size_t)2 * E * ff; }
        const float w = wts[t * wcols + e];
        float a = 0.f;
        if (w != 0.f) {
            const T* row = gu + t * (size_t)(2 * total) + base;
            const float wi = w_in ? w : 1.0f, wo = w_in ? 1.0f : w;
            const float g = fminf(to_float(row[j]) * wi, lim);
            const float u = fminf(fmaxf(to_float(row[width + j]) * wi, -lim), lim);
            a = wo * (g / (1.0f + expf(-alpha * g))) * (u + up_add);
        }
        out[i] = from_float<T>(a);
    }
}

// The same, 16 bytes of columns a thread (the experts' widths are multiples of that many columns, so a thread's
// columns belong to one expert): gate and up are read 16 bytes at a time, the result is written so.
template <typename T>
__global__ void __launch_bounds__(256)
moe_expert_act_vec_kernel(const T* __restrict__ gu, const float* __restrict__ wts, int E, int ff, float limit, int shared_ff,
                          float shared_limit, float alpha, T* __restrict__ out, int T_rows, int wcols, float up_add, int w_in) {
    constexpr int V = Vec16<T>::N;
    const int total = E * ff + shared_ff, per_row = total / V;
    grid_dependents_launch();
    grid_dependency_wait();
    for (int t = blockIdx.y; t < T_rows; t += gridDim.y) {
        const float* wrow = wts + (size_t)t * wcols;
        const T* grow = gu + (size_t)t * (2 * (size_t)total);
        T* orow = out + (size_t)t * total;
        for (int ch = blockIdx.x * blockDim.x + threadIdx.x; ch < per_row; ch += gridDim.x * blockDim.x) {
            const int col = ch * V;
            int e, j, width;
            float lim;
            size_t base;
            if (col < E * ff) { e = col / ff; j = col - e * ff; width = ff; lim = limit; base = (size_t)2 * e * ff; }
            else { e = E; j = col - E * ff; width = shared_ff; lim = shared_limit; base = (size_t)2 * E * ff; }
            const float w = wrow[e];
            float a[V];
#pragma unroll
            for (int i = 0; i < V; ++i) a[i] = 0.f;
            if (w != 0.f) {
                float gv[V], uv[V];
                Vec16<T>::load(grow + base + j, gv);
                Vec16<T>::load(grow + base + width + j, uv);
                const float wi = w_in ? w : 1.0f, wo = w_in ? 1.0f : w;
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    const float g = fminf(gv[i] * wi, lim);
                    const float u = fminf(fmaxf(uv[i] * wi, -lim), lim);
                    a[i] = wo * (g / (1.0f + expf(-alpha * g))) * (u + up_add);
                }
            }
            Vec16<T>::store(orow + col, a);
        }
    }
}

// x[t, col] = w[t, e] relu(x[t, col])^2 in place over the columns of all experts side by side (expert e: `ff` columns; then
// the shared expert's `shared_ff`, whose weight is column E of the weights or, without one (shared_col == 0), 1).
// Experts of weight 0 give exact zeros.  VEC: 16 bytes of columns a thread, all of one expert.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
moe_relu2_kernel(T* __restrict__ x, const float* __restrict__ wts, int E, int ff, int shared_ff, int shared_col, int T_rows,
                 int wcols) {
    constexpr int V = VEC ? Vec16<T>::N : 1;
    const int total = E * ff + shared_ff, per_row = total / V;
    grid_dependents_launch();
    grid_dependency_wait();
    for (int t = blockIdx.y; t < T_rows; t += gridDim.y) {
        const float* wrow = wts + (size_t)t * wcols;
        T* row = x + (size_t)t * total;
        for (int ch = blockIdx.x * blockDim.x + threadIdx.x; ch < per_row; ch += gridDim.x * blockDim.x) {
            const int col = ch * V;
            const float w = col < E * ff ? wrow[col / ff] : (shared_col ? wrow[E] : 1.f);
            float a[V];
            if constexpr (VEC) {
                if (w != 0.f) Vec16<T>::load(row + col, a);
#pragma unroll
                for (int i = 0; i < V; ++i) a[i] = w != 0.f && a[i] > 0.f ? w * a[i] * a[i] : 0.f;
                Vec16<T>::store(row + col, a);
            } else {
                const float v = to_float(row[col]);
                row[col] = from_float<T>(w != 0.f && v > 0.f ? w * v * v : 0.f);
            }
        }
    }
}

// dst[t, d_off + c] = scale * x[t, c] * sigmoid(rows[t, g_off + c / per]) (no gate where rows is null): an attention's
// heads on their way into the input of an output product that other branches share.  VEC: 16 bytes a thread (per == 1).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
gate_place_kernel(const T* __restrict__ x, const T* __restrict__ rows, int row_elems, int g_off, int per, T* __restrict__ dst,
                  int dst_elems, int d_off, float scale, int width, size_t n) {
    constexpr int V = VEC ? Vec16<T>::N : 1;
    grid_dependents_launch();
    grid_dependency_wait();
    for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V) {
        const size_t t = i / width;
        const int c = (int)(i % width);
        if constexpr (VEC) {
            float a[V], g[V];
            Vec16<T>::load(x + i, a);
            if (rows != nullptr) {
                Vec16<T>::load(rows + t * row_elems + g_off + c, g);
#pragma unroll
                for (int e = 0; e < V; ++e) a[e] = scale * (a[e] / (1.0f + expf(-g[e])));
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) a[e] *= scale;
            }
            Vec16<T>::store(dst + t * dst_elems + d_off + c, a);
        } else {
            float a = to_float(x[i]);
            if (rows != nullptr) a /= 1.0f + expf(-to_float(rows[t * row_elems + g_off + c / per]));
            dst[t * dst_elems + d_off + c] = from_float<T>(scale * a);
        }
    }
}

}  // namespace janis

using namespace janis;

static inline unsigned flat_grid(size_t n) {
    const size_t want = (n + 255) / 256;
    return (unsigned)(want < 148 * 16 ? (want ? want : 1) : 148 * 16);
}

JANIS_EXPORT int janis_dyt_norm(float* h, const void* res, int res_dtype, const int* rows, float alpha, const float* w,
                                const float* b, void* y, int y_dtype, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    if (res != nullptr && rows != nullptr) return fail("dyt_norm: a residual is added to all rows, not to chosen ones");
    const dim3 grid(R), block(H >= 1024 ? 256 : 128);
#define JANIS_DYT(TR, TO)                                                                                              \
    return launch_kernel("dyt_norm", dyt_norm_kernel<TR, TO>, grid, block, 0, stream, 1, h, (const TR*)res, rows, alpha, w, \
                         b, (TO*)y, H);
    const int rd = res != nullptr ? res_dtype : JANIS_F32;
    if (rd == JANIS_F32 && y_dtype == JANIS_F32) { JANIS_DYT(float, float) }
    if (rd == JANIS_F32 && y_dtype == JANIS_BF16) { JANIS_DYT(float, bf16) }
    if (rd == JANIS_BF16 && y_dtype == JANIS_F32) { JANIS_DYT(bf16, float) }
    if (rd == JANIS_BF16 && y_dtype == JANIS_BF16) { JANIS_DYT(bf16, bf16) }
#undef JANIS_DYT
    return fail("dyt_norm: unknown dtypes %d, %d", res_dtype, y_dtype);
}

JANIS_EXPORT int janis_rmsnorm_accumulate(const void* x, int dtype, const float* w, float eps, float share, float* acc,
                                          int first, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    const dim3 grid(R), block(H >= 1024 ? 256 : 128);
    if (dtype == JANIS_F32)
        return launch_kernel("rmsnorm_accumulate", rmsnorm_accumulate_kernel<float>, grid, block, 0, stream, 1,
                             (const float*)x, w, eps, share, acc, first, H);
    if (dtype == JANIS_BF16)
        return launch_kernel("rmsnorm_accumulate", rmsnorm_accumulate_kernel<bf16>, grid, block, 0, stream, 1,
                             (const bf16*)x, w, eps, share, acc, first, H);
    return fail("rmsnorm_accumulate: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_sigmoid_gate(void* x, const void* rows, int dtype, int row_elems, int g_off, int T, int width,
                                    int per, cudaStream_t stream) {
    if (T <= 0 || width <= 0) return 0;
    if (per <= 0 || width % per) return fail("sigmoid_gate: runs of %d elements do not divide %d", per, width);
    if (g_off < 0 || g_off + width / per > row_elems) return fail("sigmoid_gate: %d gates at %d do not fit rows of %d", width / per, g_off, row_elems);
    const size_t n = (size_t)T * width;
    if (dtype == JANIS_F32)
        return launch_kernel("sigmoid_gate", sigmoid_gate_kernel<float>, dim3(flat_grid(n)), dim3(256), 0, stream, 1, (float*)x,
                             (const float*)rows, row_elems, g_off, width, per, n);
    if (dtype == JANIS_BF16)
        return launch_kernel("sigmoid_gate", sigmoid_gate_kernel<bf16>, dim3(flat_grid(n)), dim3(256), 0, stream, 1, (bf16*)x,
                             (const bf16*)rows, row_elems, g_off, width, per, n);
    return fail("sigmoid_gate: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_group_norm(float* h, const void* res, int res_dtype, const int* rows, float alpha, const float* w,
                                  float eps, int groups, void* y, int y_dtype, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    if (groups <= 0 || H % groups) return fail("group_norm: %d groups do not divide a row of %d", groups, H);
    if (res != nullptr && rows != nullptr) return fail("group_norm: a residual is added to all rows, not to chosen ones");
    if (res == nullptr && y == nullptr) return fail("group_norm: nothing to write");
    const size_t bytes = ((size_t)H + groups + 32) * sizeof(float);
    if (bytes > 200 * 1024) return fail("group_norm: a row of %d does not fit shared memory", H);
    const dim3 grid(R), block(H >= 1024 ? 256 : 128);
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = (H / groups) % 4 == 0 && aligned(h) && aligned(res) && aligned(w) && aligned(y);
#define JANIS_GN_V(TR, TO, VEC)                                                                                        \
    {                                                                                                                  \
        static size_t most = 0;                                                                                        \
        if (bytes > most && bytes > 48 * 1024) {                                                                       \
            cudaError_t e = cudaFuncSetAttribute(group_norm_kernel<TR, TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes); \
            if (e != cudaSuccess) return fail("group_norm: shared memory of %zu bytes refused: %s", bytes, cudaGetErrorString(e)); \
            most = bytes;                                                                                              \
        }                                                                                                              \
        return launch_kernel("group_norm", group_norm_kernel<TR, TO, VEC>, grid, block, bytes, stream, 1, h, (const TR*)res, rows, \
                             alpha, w, eps, groups, (TO*)y, H);                                                        \
    }
#define JANIS_GN(TR, TO)                                                                                               \
    {                                                                                                                  \
        if (vec) JANIS_GN_V(TR, TO, true)                                                                              \
        JANIS_GN_V(TR, TO, false)                                                                                      \
    }
    const int rd = res != nullptr ? res_dtype : JANIS_F32, yd = y != nullptr ? y_dtype : JANIS_F32;
    if (rd == JANIS_F32 && yd == JANIS_F32) JANIS_GN(float, float)
    if (rd == JANIS_F32 && yd == JANIS_BF16) JANIS_GN(float, bf16)
    if (rd == JANIS_BF16 && yd == JANIS_F32) JANIS_GN(bf16, float)
    if (rd == JANIS_BF16 && yd == JANIS_BF16) JANIS_GN(bf16, bf16)
#undef JANIS_GN
#undef JANIS_GN_V
    return fail("group_norm: unknown dtypes %d, %d", res_dtype, y_dtype);
}

template <typename TR, typename TO>
static int stream_norm_launch(float* h, const void* r0, const void* r1, const StreamSum& s, const float* w_next, float eps_next,
                              int centred, void* y, const int* rows, int R, int H, bool vec, cudaStream_t stream) {
#define JANIS_SN(VW, VPT, NT)                                                                                          \
    return launch_kernel("stream_norm", stream_norm_kernel<TR, TO, VW, VPT>, dim3(R), dim3(NT), 0, stream, 1, h, (const TR*)r0, \
                         (const TR*)r1, s, w_next, eps_next, centred, (TO*)y, rows, H);
    if (vec) {
        const int pieces = H / 4;
        if (pieces <= 128) { JANIS_SN(4, 1, 128) }
        if (pieces <= 256) { JANIS_SN(4, 1, 256) }
        if (pieces <= 384) { JANIS_SN(4, 3, 128) }
        if (pieces <= 512) { JANIS_SN(4, 2, 256) }
        if (pieces <= 768) { JANIS_SN(4, 3, 256) }
        if (pieces <= 1024) { JANIS_SN(4, 4, 256) }
        if (pieces <= 1536) { JANIS_SN(4, 6, 256) }
    }
    JANIS_SN(1, 1, H >= 1024 ? 256 : 128)
#undef JANIS_SN
}

JANIS_EXPORT int janis_stream_norm(float* h, const void* r0, const void* r1, int r_dtype, const float* w0, const float* w1, float eps,
                                   float share, const float* scale, const float* more, const float* w_next, float eps_next,
                                   int centred, void* y, int y_dtype, const int* rows, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    if (r0 != nullptr && rows != nullptr) return fail("stream_norm: a result is added to all rows, not to chosen ones");
    if (r0 == nullptr && (r1 != nullptr || more != nullptr || w_next == nullptr)) return fail("stream_norm: nothing to do, or a second branch without a first");
    if ((w0 == nullptr) != (w1 == nullptr) && r1 != nullptr) return fail("stream_norm: both branches are normed, or none");
    if (r1 != nullptr && w0 == nullptr) return fail("stream_norm: two branches are normed before they are added");
    if (w_next != nullptr && y == nullptr) return fail("stream_norm: a norm needs an output");
    const StreamSum s = {w0, w1, eps, share, scale, more};
    const uintptr_t all = (uintptr_t)h | (uintptr_t)r0 | (uintptr_t)r1 | (uintptr_t)w0 | (uintptr_t)w1 | (uintptr_t)scale |
                          (uintptr_t)more | (uintptr_t)w_next | (uintptr_t)y;
    const bool vec = H % 4 == 0 && (all & 15) == 0;
    const int rd = r0 != nullptr ? r_dtype : JANIS_F32, yd = y != nullptr ? y_dtype : JANIS_F32;
#define JANIS_SNT(TR, TO) return stream_norm_launch<TR, TO>(h, r0, r1, s, w_next, eps_next, centred, y, rows, R, H, vec, stream);
    if (rd == JANIS_F32 && yd == JANIS_F32) { JANIS_SNT(float, float) }
    if (rd == JANIS_F32 && yd == JANIS_BF16) { JANIS_SNT(float, bf16) }
    if (rd == JANIS_BF16 && yd == JANIS_F32) { JANIS_SNT(bf16, float) }
    if (rd == JANIS_BF16 && yd == JANIS_BF16) { JANIS_SNT(bf16, bf16) }
#undef JANIS_SNT
    return fail("stream_norm: unknown dtypes %d, %d", r_dtype, y_dtype);
}

JANIS_EXPORT int janis_round_rows(const float* h, void* y, size_t n, cudaStream_t stream) {
    if (n == 0) return 0;
    return launch_kernel("round_rows", round_rows_kernel, dim3(flat_grid(n)), dim3(256), 0, stream, 1, h, (bf16*)y, n);
}

JANIS_EXPORT int janis_moe_route(const float* z, const float* correction, int T, int E, int n_groups, int keep, int top,
                                 float scale, int shared_gate, float* out, int n_identity, int softmax, int group_best, int raw,
                                 cudaStream_t stream) {
    if (T <= 0) return 0;
    const int N = E + n_identity;
    if (E < 0 || n_identity < 0 || N <= 0 || N > 1024) return fail("moe_route: %d experts and %d identity entries (up to 1024 are taken)", E, n_identity);
    if (n_identity > 0 && n_groups != 1) return fail("moe_route: identity entries stand in no group");
    if (n_groups <= 0 || N % n_groups || keep <= 0 || keep > n_groups || top <= 0 || top > keep * (N / n_groups))
        return fail("moe_route: %d entries in %d groups, %d kept, %d chosen", N, n_groups, keep, top);
    const size_t bytes = (size_t)ROUTE_WARPS * 4 * N * sizeof(float);
    return launch_kernel("moe_route", moe_route_kernel, dim3((T + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32),
                         bytes, stream, 1, z, correction, T, E, n_groups, keep, top, scale, shared_gate, out, n_identity, softmax, group_best, raw);
}

JANIS_EXPORT int janis_moe_identity_add(void* out, const void* y, int dtype, const float* wts, int wts_stride, int w_col, int T,
                                        int width, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (w_col < 0 || w_col >= wts_stride) return fail("moe_identity_add: column %d of %d", w_col, wts_stride);
    const size_t n = (size_t)T * width;
    if (dtype == JANIS_F32)
        return launch_kernel("moe_identity_add", moe_identity_add_kernel<float>, dim3(flat_grid(n)), dim3(256), 0, stream, 1,
                             (float*)out, (const float*)y, wts, wts_stride, w_col, width, n);
    if (dtype == JANIS_BF16)
        return launch_kernel("moe_identity_add", moe_identity_add_kernel<bf16>, dim3(flat_grid(n)), dim3(256), 0, stream, 1,
                             (bf16*)out, (const bf16*)y, wts, wts_stride, w_col, width, n);
    return fail("moe_identity_add: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_moe_expert_act(const void* gu, int dtype, const float* wts, int E, int ff, float limit, int shared_ff,
                                      float shared_limit, float alpha, void* out, int T, int wts_stride, float up_add,
                                      int w_in, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (wts_stride <= 0) wts_stride = E + (shared_ff ? 1 : 0);
    const size_t n = (size_t)T * ((size_t)E * ff + shared_ff);
    const int v = dtype == JANIS_F32 ? 4 : 8;
    if (ff % v == 0 && shared_ff % v == 0 && (((uintptr_t)gu | (uintptr_t)out) & 15) == 0) {
        const int per_row = (E * ff + shared_ff) / v;
        const dim3 grid((per_row + 255) / 256, T < 65535 ? T : 65535), block(256);
        if (dtype == JANIS_F32)
            return launch_kernel("moe_expert_act", moe_expert_act_vec_kernel<float>, grid, block, 0, stream, 1, (const float*)gu,
                                 wts, E, ff, limit, shared_ff, shared_limit, alpha, (float*)out, T, wts_stride, up_add, w_in);
        if (dtype == JANIS_BF16)
            return launch_kernel("moe_expert_act", moe_expert_act_vec_kernel<bf16>, grid, block, 0, stream, 1, (const bf16*)gu,
                                 wts, E, ff, limit, shared_ff, shared_limit, alpha, (bf16*)out, T, wts_stride, up_add, w_in);
    }
    if (dtype == JANIS_F32)
        return launch_kernel("moe_expert_act", moe_expert_act_kernel<float>, dim3(flat_grid(n)), dim3(256), 0, stream, 1,
                             (const float*)gu, wts, E, ff, limit, shared_ff, shared_limit, alpha, (float*)out, n, wts_stride, up_add, w_in);
    if (dtype == JANIS_BF16)
        return launch_kernel("moe_expert_act", moe_expert_act_kernel<bf16>, dim3(flat_grid(n)), dim3(256), 0, stream, 1,
                             (const bf16*)gu, wts, E, ff, limit, shared_ff, shared_limit, alpha, (bf16*)out, n, wts_stride, up_add, w_in);
    return fail("moe_expert_act: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_moe_relu2(void* x, int dtype, const float* wts, int wts_stride, int E, int ff, int shared_ff,
                                 int shared_col, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    const int total = E * ff + shared_ff;
    if (total <= 0) return fail("moe_relu2: no columns (%d experts of %d, shared %d)", E, ff, shared_ff);
    if (E + (shared_col ? 1 : 0) > wts_stride) return fail("moe_relu2: %d weights a row for %d experts", wts_stride, E);
    const int v = dtype == JANIS_F32 ? 4 : 8;
    const bool vec = ff % v == 0 && shared_ff % v == 0 && ((uintptr_t)x & 15) == 0;
    const int per_row = vec ? total / v : total;
    const dim3 grid((per_row + 255) / 256, T < 65535 ? T : 65535), block(256);
#define JANIS_RELU2(TT, VEC)                                                                                           \
    return launch_kernel("moe_relu2", moe_relu2_kernel<TT, VEC>, grid, block, 0, stream, 1, (TT*)x, wts, E, ff, shared_ff, \
                         shared_col, T, wts_stride);
    if (dtype == JANIS_F32) {
        if (vec) JANIS_RELU2(float, true)
        JANIS_RELU2(float, false)
    }
    if (dtype == JANIS_BF16) {
        if (vec) JANIS_RELU2(bf16, true)
        JANIS_RELU2(bf16, false)
    }
#undef JANIS_RELU2
    return fail("moe_relu2: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_gate_place(const void* x, const void* rows, int dtype, int row_elems, int g_off, int per, void* dst,
                                  int dst_elems, int d_off, float scale, int T, int width, cudaStream_t stream) {
    if (T <= 0 || width <= 0) return 0;
    if (per <= 0 || width % per) return fail("gate_place: runs of %d elements do not divide %d", per, width);
    if (rows != nullptr && (g_off < 0 || g_off + width / per > row_elems)) return fail("gate_place: %d gates at %d do not fit rows of %d", width / per, g_off, row_elems);
    if (d_off < 0 || d_off + width > dst_elems) return fail("gate_place: %d columns at %d do not fit rows of %d", width, d_off, dst_elems);
    const size_t n = (size_t)T * width;
    const int v = dtype == JANIS_F32 ? 4 : 8;
    const bool vec = width % v == 0 && d_off % v == 0 && dst_elems % v == 0 && (((uintptr_t)x | (uintptr_t)dst) & 15) == 0 &&
                     (rows == nullptr || (per == 1 && g_off % v == 0 && row_elems % v == 0 && ((uintptr_t)rows & 15) == 0));
#define JANIS_PLACE(TT, VEC)                                                                                           \
    return launch_kernel("gate_place", gate_place_kernel<TT, VEC>, dim3(flat_grid(VEC ? n / v : n)), dim3(256), 0, stream, 1, \
                         (const TT*)x, (const TT*)rows, row_elems, g_off, per, (TT*)dst, dst_elems, d_off, scale, width, n);
    if (dtype == JANIS_F32) {
        if (vec) JANIS_PLACE(float, true)
        JANIS_PLACE(float, false)
    }
    if (dtype == JANIS_BF16) {
        if (vec) JANIS_PLACE(bf16, true)
        JANIS_PLACE(bf16, false)
    }
#undef JANIS_PLACE
    return fail("gate_place: unknown dtype %d", dtype);
}
