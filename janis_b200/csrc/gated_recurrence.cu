// The gated linear recurrence of a recurrent block: one number of state per channel, a decay that the input chooses.
//
//   r = sigmoid(zr + br),  i = sigmoid(zi + bi)          zr, zi: a square product per block of channels of u (float)
//   log a = decay * r                                    decay < 0, a number per channel
//   S <- a S + sqrt(1 - a^2) i u                         S starts at zero, lives in the cache as floats
//   out = scale * S * gelu_tanh(y + yb)                  y: another projection of the block's input
//
// Everything between u and out is float.  A channel that remembers thousands of tokens has a just below 1, where a float
// holds a to 6e-8 only; so a - 1 = expm1(log a) is what is kept, the step is S + (S (a - 1) + input), and
// 1 - a^2 = -(a - 1)(a + 1) loses nothing.  Two kernels: one for steps that bring several tokens (the gates' products are
// formed before it), one for steps of single rows, which forms the gates' products itself.
// Sequences without a slot (padding) start from zero and store nothing.
#include "common.cuh"

namespace janis {

__device__ __forceinline__ float logistic(float v) { return 1.0f / (1.0f + expf(-v)); }

// one token's decay minus one and input
__device__ __forceinline__ void recurrence_terms(float zr, float zi, float u, float decay, float& am1, float& in) {
    am1 = expm1f(decay * logistic(zr));
    in = sqrtf(fmaxf(-am1 * (am1 + 2.0f), 0.f)) * logistic(zi) * u;
}

struct RecurrenceShape {
    int C, block;                 // channels; channels a block of the gates' products
    long long g_tok, g_block;     // elements between neighbouring tokens' and blocks' gate logits (r's of a block, then i's)
    int y_stride, y_off;          // y[t, c] = y_rows[t * y_stride + y_off + c]
    int o_stride, o_off;          // out[t * o_stride + o_off + c]
    float scale;
};

// A CTA per (CH channels, sequence).  Its NT / CH groups of threads take runs of TT tokens: each runs its tokens from a
// state of zero, keeping every token's state and the product of the decays so far (minus one); the groups' totals meet in
// shared memory (two buffers that take turns, one barrier a round), every thread carries the state over all groups in
// order and puts the state that enters its own group under its tokens.  The inputs of the next round are on their way
// while this one is computed.
template <typename T, int CH, int TT, int NT>
__global__ void __launch_bounds__(NT)
gated_recurrence_scan_kernel(const T* __restrict__ u, const float* __restrict__ gates, const float* __restrict__ br,
                             const float* __restrict__ bi, const float* __restrict__ decay, const T* __restrict__ y_rows,
                             const float* __restrict__ yb, RecurrenceShape g, const int* __restrict__ seq_slot,
                             const int* __restrict__ seq_first_row, const int* __restrict__ seq_start,
                             const int* __restrict__ seq_end, float* __restrict__ state, T* __restrict__ out) {
    constexpr int NG = NT / CH, ROUND = NG * TT;
    __shared__ float2 tot_s[2][NG][CH];
    const int tid = threadIdx.x, cl = tid % CH, grp = tid / CH, seq = blockIdx.y;
    const int c_raw = blockIdx.x * CH + cl;
    const bool live = c_raw < g.C;
    const int c = live ? c_raw : g.C - 1;
    grid_dependents_launch();
    const int slot = seq_slot[seq], row0 = seq_first_row[seq], n_tok = seq_end[seq] - seq_start[seq];
    if (n_tok <= 0) return;
    const float brc = br[c], bic = bi[c], dec = decay[c], ybc = yb != nullptr ? yb[c] : 0.f;
    grid_dependency_wait();
    const T* pu = u + (size_t)row0 * g.C + c;
    const float* pg = gates + (size_t)row0 * g.g_tok + (size_t)(c / g.block) * g.g_block + c % g.block;
    const T* py = y_rows + (size_t)row0 * g.y_stride + g.y_off + c;
    T* po = out + (size_t)row0 * g.o_stride + g.o_off + c;
    float* st = slot >= 0 ? state + (size_t)slot * g.C + c : nullptr;
    float S = st != nullptr ? *st : 0.f;
    struct Round { float u[TT], zr[TT], zi[TT], y[TT]; };
    auto fetch = [&](int t0, Round& x) {
#pragma unroll
        for (int k = 0; k < TT; ++k) {
            const size_t t = (size_t)min(t0 + grp * TT + k, n_tok - 1);
            x.u[k] = to_float(pu[t * g.C]);
            x.zr[k] = pg[t * g.g_tok];
            x.zi[k] = pg[t * g.g_tok + g.block];
            x.y[k] = to_float(py[t * g.y_stride]);
        }
    };
    Round cur, nxt;
    fetch(0, cur);
    for (int t0 = 0, buf = 0; t0 < n_tok; t0 += ROUND, buf ^= 1) {
        if (t0 + ROUND < n_tok) fetch(t0 + ROUND, nxt);
        float own[TT], keep[TT];            // the token's state from zero; the decays' product up to it, minus one
        float B = 0.f, A = 0.f;
#pragma unroll
        for (int k = 0; k < TT; ++k) {
            float am1, in;
            recurrence_terms(cur.zr[k] + brc, cur.zi[k] + bic, cur.u[k], dec, am1, in);
            if (t0 + grp * TT + k >= n_tok) am1 = in = 0.f;      // (beyond the end nothing changes)
            B = B + fmaf(B, am1, in);
            A = A + fmaf(A, am1, am1);
            own[k] = B;
            keep[k] = A;
        }
        tot_s[buf][grp][cl] = make_float2(A, B);
        __syncthreads();
        float enter = S;
#pragma unroll 8
        for (int q = 0; q < NG; ++q) {
            if (q == grp) enter = S;
            const float2 ab = tot_s[buf][q][cl];
            S = S + fmaf(S, ab.x, ab.y);
        }
#pragma unroll
        for (int k = 0; k < TT; ++k) {
            const int t = t0 + grp * TT + k;
            if (t < n_tok && live)
                po[(size_t)t * g.o_stride] = from_float<T>(g.scale * (own[k] + fmaf(enter, keep[k], enter)) * gelu_tanh(cur.y[k] + ybc));
        }
        cur = nxt;
    }
    if (st != nullptr && live && grp == 0) *st = S;
}

// Steps of single rows (every sequence brings one token).  A CTA per (block of channels, 16 channels of it, 8 rows): the
// rows' u of the block in shared memory as floats; 8 lanes share a channel, take its two rows of the gates' matrices 16
// bytes at a time in turn (the first pieces before the kernel waits for its predecessor: weights are constants) and scatter
// their partial sums so that lane r of the eight ends up with row r's, which it finishes.
constexpr int REC_ROWS = 8, REC_WARPS = 4, REC_CHANNELS = REC_WARPS * 4;

// v[0..7] of each of 8 lanes: the lanes' sums of v[own lane], in a fixed order
__device__ __forceinline__ float scatter_sum8(float (&v)[REC_ROWS], int sub) {
#pragma unroll
    for (int half = 4; half >= 1; half >>= 1) {
        const bool up = (sub & half) != 0;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if (i < half) {
                const float mine = up ? v[i + half] : v[i], other = up ? v[i] : v[i + half];
                v[i] = mine + __shfl_xor_sync(0xffffffffu, other, half);
            }
        }
    }
    return v[0];
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(REC_WARPS * 32)
gated_recurrence_rows_kernel(const T* __restrict__ u, const T* __restrict__ w, const float* __restrict__ br,
                             const float* __restrict__ bi, const float* __restrict__ decay, const T* __restrict__ y_rows,
                             const float* __restrict__ yb, RecurrenceShape g, const int* __restrict__ tok_seq,
                             const int* __restrict__ seq_slot, int n_rows, float* __restrict__ state, T* __restrict__ out) {
    constexpr int V = Vec16<T>::N, AHEAD = 4;             // pieces asked for together
    extern __shared__ __align__(16) float rec_u[];        // [REC_ROWS][block]
    const int tid = threadIdx.x, lane = tid & 31, sub = lane & 7, n = g.block;
    const int b = blockIdx.x, j_raw = blockIdx.y * REC_CHANNELS + (tid >> 3), row0 = blockIdx.z * REC_ROWS;
    const int here = min(REC_ROWS, n_rows - row0);
    const bool mine = j_raw < n;
    const int j = mine ? j_raw : n - 1, c = b * n + j;    // (lanes without a channel repeat the last one and store nothing)
    const T* wr = w + ((size_t)b * 2 * n + j) * n;
    const T* wi = wr + (size_t)n * n;
    const bool live = mine && sub < here;
    const int row = row0 + (sub < here ? sub : 0);
    grid_dependents_launch();
    uint4 pr[AHEAD], pi[AHEAD];
    if (VEC) {
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            const int k = (sub + 8 * a) * V;
            if (k < n) {
                pr[a] = *reinterpret_cast<const uint4*>(wr + k);
                pi[a] = *reinterpret_cast<const uint4*>(wi + k);
            }
        }
    }
    const float brc = br[c], bic = bi[c], dec = decay[c], ybc = yb != nullptr ? yb[c] : 0.f;
    const int slot = live ? seq_slot[tok_seq[row]] : -1;
    grid_dependency_wait();
    const float S0 = slot >= 0 ? state[(size_t)slot * g.C + c] : 0.f;
    const float y = to_float(y_rows[(size_t)row * g.y_stride + g.y_off + c]);
    if (VEC) {
        const int per = n / V;
        for (int k = tid; k < REC_ROWS * per; k += REC_WARPS * 32) {
            const int r = k / per, at = (k - r * per) * V;
            float x[V];
            if (r < here) Vec16<T>::load(u + (size_t)(row0 + r) * g.C + (size_t)b * n + at, x);
#pragma unroll
            for (int e = 0; e < V; e += 4) {
                if (r >= here) x[e] = x[e + 1] = x[e + 2] = x[e + 3] = 0.f;
                Vec16<float>::store(rec_u + r * n + at + e, x + e);
            }
        }
    } else {
        for (int k = tid; k < REC_ROWS * n; k += REC_WARPS * 32) {
            const int r = k / n;
            rec_u[k] = r < here ? to_float(u[(size_t)(row0 + r) * g.C + (size_t)b * n + k % n]) : 0.f;
        }
    }
    __syncthreads();
    float ar[REC_ROWS], ai[REC_ROWS];
#pragma unroll
    for (int r = 0; r < REC_ROWS; ++r) ar[r] = ai[r] = 0.f;
    if (VEC) {
        for (int k0 = 0; k0 < n; k0 += 8 * V * AHEAD) {
#pragma unroll
            for (int a = 0; a < AHEAD; ++a) {
                const int k = k0 + (sub + 8 * a) * V;
                if (k < n) {
                    float fr[V], fi[V];
                    Vec16<T>::load(reinterpret_cast<const T*>(&pr[a]), fr);
                    Vec16<T>::load(reinterpret_cast<const T*>(&pi[a]), fi);
#pragma unroll
                    for (int r = 0; r < REC_ROWS; ++r) {
#pragma unroll
                        for (int e = 0; e < V; e += 4) {
                            float x[4];
                            Vec16<float>::load(rec_u + r * n + k + e, x);
#pragma unroll
                            for (int q = 0; q < 4; ++q) {
                                ar[r] = fmaf(fr[e + q], x[q], ar[r]);
                                ai[r] = fmaf(fi[e + q], x[q], ai[r]);
                            }
                        }
                    }
                }
                const int kn = k + 8 * V * AHEAD;             // the piece of the next round takes this one's place
                if (kn < n) {
                    pr[a] = *reinterpret_cast<const uint4*>(wr + kn);
                    pi[a] = *reinterpret_cast<const uint4*>(wi + kn);
                }
            }
        }
    } else {
        for (int k = sub; k < n; k += 8) {
            const float x0 = to_float(wr[k]), x1 = to_float(wi[k]);
#pragma unroll
            for (int r = 0; r < REC_ROWS; ++r) {
                ar[r] = fmaf(x0, rec_u[r * n + k], ar[r]);
                ai[r] = fmaf(x1, rec_u[r * n + k], ai[r]);
            }
        }
    }
    const float zr = scatter_sum8(ar, sub), zi = scatter_sum8(ai, sub);
    if (!live) return;
    float am1, in;
    recurrence_terms(zr + brc, zi + bic, to_float(u[(size_t)row * g.C + c]), dec, am1, in);
    const float S = S0 + fmaf(S0, am1, in);
    if (slot >= 0) state[(size_t)slot * g.C + c] = S;
    out[(size_t)row * g.o_stride + g.o_off + c] = from_float<T>(g.scale * S * gelu_tanh(y + ybc));
}

}  // namespace janis

using namespace janis;

static int recurrence_check(const char* what, int C, int block, int y_stride, int y_off, int o_stride, int o_off) {
    if (C <= 0 || block <= 0 || C % block) return fail("%s: %d channels do not divide into blocks of %d", what, C, block);
    if (y_off < 0 || y_off + C > y_stride) return fail("%s: %d channels at %d do not fit rows of %d", what, C, y_off, y_stride);
    if (o_off < 0 || o_off + C > o_stride) return fail("%s: %d channels at %d do not fit result rows of %d", what, C, o_off, o_stride);
    return 0;
}

JANIS_EXPORT int janis_gated_recurrence_scan(const void* u, int dtype, const float* gates, long long g_tok, long long g_block,
                                             const float* br, const float* bi, const float* decay, const void* y_rows,
                                             int y_stride, int y_off, const float* yb, const int* seq_slot,
                                             const int* seq_first_row, const int* seq_start, const int* seq_end, int n_seq,
                                             float* state, void* out, int o_stride, int o_off, float scale, int C, int block,
                                             cudaStream_t stream) {
    if (n_seq <= 0) return 0;
    if (recurrence_check("gated_recurrence_scan", C, block, y_stride, y_off, o_stride, o_off)) return 1;
    if (n_seq > 65535) return fail("gated_recurrence_scan: too many sequences (%d)", n_seq);
    const RecurrenceShape g = {C, block, g_tok, g_block, y_stride, y_off, o_stride, o_off, scale};
    // narrow CTAs while wide ones would leave SMs idle
    const bool narrow = (long long)n_seq * ((C + 31) / 32) < 2 * 148;
#define JANIS_REC(T, CH, TT, NT)                                                                                       \
    return launch_kernel("gated_recurrence_scan", gated_recurrence_scan_kernel<T, CH, TT, NT>, dim3((C + CH - 1) / CH, n_seq), \
                         dim3(NT), 0, stream, 1, (const T*)u, gates, br, bi, decay, (const T*)y_rows, yb, g,  \
                         seq_slot, seq_first_row, seq_start, seq_end, state, (T*)out);
    if (dtype == JANIS_F32) {
        if (narrow) JANIS_REC(float, 16, 4, 512)
        JANIS_REC(float, 32, 4, 256)
    }
    if (dtype == JANIS_BF16) {
        if (narrow) JANIS_REC(bf16, 16, 4, 512)
        JANIS_REC(bf16, 32, 4, 256)
    }
#undef JANIS_REC
    return fail("gated_recurrence_scan: unknown dtype %d", dtype);
}

JANIS_EXPORT int janis_gated_recurrence_rows(const void* u, int dtype, const void* w, const float* br, const float* bi,
                                             const float* decay, const void* y_rows, int y_stride, int y_off, const float* yb,
                                             const int* tok_seq, const int* seq_slot, int n_rows, float* state, void* out,
                                             int o_stride, int o_off, float scale, int C, int block, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (recurrence_check("gated_recurrence_rows", C, block, y_stride, y_off, o_stride, o_off)) return 1;
    const size_t bytes = (size_t)REC_ROWS * block * sizeof(float);
    if (bytes > 48 * 1024) return fail("gated_recurrence_rows: blocks of %d channels do not fit shared memory", block);
    const int blocks = C / block, gy = (block + REC_CHANNELS - 1) / REC_CHANNELS, gz = (n_rows + REC_ROWS - 1) / REC_ROWS;
    if (gy > 65535 || gz > 65535) return fail("gated_recurrence_rows: %d rows, blocks of %d", n_rows, block);
    const RecurrenceShape g = {C, block, 0, 0, y_stride, y_off, o_stride, o_off, scale};
    const int v = dtype == JANIS_F32 ? 4 : 8;
    const bool vec = block % v == 0 && ((uintptr_t)w & 15) == 0;
#define JANIS_REC(T, VEC)                                                                                              \
    return launch_kernel("gated_recurrence_rows", gated_recurrence_rows_kernel<T, VEC>, dim3(blocks, gy, gz),          \
                         dim3(REC_WARPS * 32), bytes, stream, 1, (const T*)u, (const T*)w, br, bi, decay, (const T*)y_rows, \
                         yb, g, tok_seq, seq_slot, n_rows, state, (T*)out);
    if (dtype == JANIS_F32) {
        if (vec) JANIS_REC(float, true)
        JANIS_REC(float, false)
    }
    if (dtype == JANIS_BF16) {
        if (vec) JANIS_REC(bf16, true)
        JANIS_REC(bf16, false)
    }
#undef JANIS_REC
    return fail("gated_recurrence_rows: unknown dtype %d", dtype);
}
