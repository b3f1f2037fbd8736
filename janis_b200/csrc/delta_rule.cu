// The gated delta rule: a recurrent mixer with a matrix of state per head that is corrected towards each value.
//
//   k, q  unit vectors per key head (x / sqrt(sum(x^2) + 1e-6); q also times q_scale), both shared by H / G heads
//   beta = sigmoid(zb),   g = exp(decay * softplus(za + dt_bias))         decay < 0; one of each per head
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q       S: [d, dv] float, starts at zero
//
// Everything from the convolved projections on is float.  The state lives in the cache as S^T ([dv, d] per head and
// slot): a column's key channels lie side by side.  Sequences without a slot (padding) start from zero and store nothing.
//
// Steps of several tokens take the tokens of a sequence four at a time.  With G_i = g_1 .. g_i and c_ij = g_{j+1} .. g_i
// inside such a block, and S the state before it,
//
//   u_i = beta_i (v_i - G_i S^T k_i - sum_{j<i} c_ij (k_j . k_i) u_j)
//   o_i = G_i S^T q_i + sum_{j<=i} c_ij (k_j . q_i) u_j
//   S  <- G_4 S + sum_j c_4j k_j u_j^T
//
// which is the recurrence itself with the sums regrouped: the eight products with S are independent of each other, and one
// exchange between the lanes of a column serves four tokens.  What does not depend on S (the norms, the products of the
// keys and queries among themselves, the decays) is formed once per block by `delta_coef` for all columns of the heads.
// A state that remembers thousands of tokens has g just below 1, where a float holds it to 6e-8 only: what the state is
// multiplied with is kept as g - 1.
#include "common.cuh"

#include <type_traits>

namespace janis {

constexpr int DELTA_KS = 16;         // lanes that share a column of the state in a prompt (each holds a run of key channels)
constexpr int DELTA_GROUPS = 8;      // such groups of lanes in a CTA
constexpr int DELTA_NT = DELTA_KS * DELTA_GROUPS;
constexpr int DELTA_BLOCK = 4;       // tokens that are taken together
constexpr int DELTA_COEF = 12;       // floats per (token, head): see delta_coef_kernel
constexpr float DELTA_UNIT_EPS = 1e-6f;

struct DeltaShape {
    int H, G, d, dv;
    int x_elems, q_off, k_off, v_off;        // the convolved rows: q [G, d], k [G, d], v [H, dv]
    int z_elems, a_off, b_off;               // the projected rows: za [H], zb [H]
    float q_scale;
};

__device__ __forceinline__ float delta_logistic(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float delta_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// g - 1 and beta of one (token, head)
template <typename T>
__device__ __forceinline__ void delta_gates(const T* __restrict__ zrow, const DeltaShape& s, int h, float decay, float dt_bias,
                                            float& gm1, float& beta) {
    gm1 = expm1f(decay * delta_softplus(to_float(zrow[s.a_off + h]) + dt_bias));
    beta = delta_logistic(to_float(zrow[s.b_off + h]));
}

// A warp per (block of up to four tokens, key head); the warp of a token that starts no block has nothing to do.  Leaves
// for every token i of the block and every head of the key head
//   [0] G_i / |k_i|   [1] beta_i   [2 .. 4] c_ij k_j.k_i (j < i)   [5 .. 8] c_ij k_j.q_i (j <= i)
//   [9] c_lj / |k_i| (l: the block's last token)   [10] G_i q_scale / |q_i|   [11] G_l - 1
// with k and q as unit vectors in the products and 0 where j is out of range; the scan then works with raw keys and queries.
template <typename T>
__global__ void __launch_bounds__(128)
delta_coef_kernel(const T* __restrict__ x, const T* __restrict__ z, DeltaShape s, const float* __restrict__ decay,
                  const float* __restrict__ dt_bias, const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_end, float* __restrict__ coef, int n_tok) {
    const int t = blockIdx.x, kvh = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    grid_dependents_launch();
    const int seq = tok_seq[t], i0 = tok_pos[t] - seq_start[seq];
    const int n = min(min(DELTA_BLOCK, seq_end[seq] - tok_pos[t]), n_tok - t);
    grid_dependency_wait();
    if (i0 % DELTA_BLOCK != 0 || kvh >= s.G || n <= 0) return;
    float kk[DELTA_BLOCK][DELTA_BLOCK], kq[DELTA_BLOCK][DELTA_BLOCK], qq[DELTA_BLOCK];      // [i][j], j <= i
#pragma unroll
    for (int i = 0; i < DELTA_BLOCK; ++i) {
        qq[i] = 0.f;
#pragma unroll
        for (int j = 0; j < DELTA_BLOCK; ++j) kk[i][j] = kq[i][j] = 0.f;
    }
#pragma unroll 2
    for (int c = lane; c < s.d; c += 32) {
        float kv[DELTA_BLOCK], qv[DELTA_BLOCK];
#pragma unroll
        for (int i = 0; i < DELTA_BLOCK; ++i) {
            kv[i] = qv[i] = 0.f;
            if (i < n) {
                const T* row = x + (size_t)(t + i) * s.x_elems + kvh * s.d + c;
                kv[i] = to_float(row[s.k_off]);
                qv[i] = to_float(row[s.q_off]);
            }
        }
#pragma unroll
        for (int i = 0; i < DELTA_BLOCK; ++i) {
            qq[i] = fmaf(qv[i], qv[i], qq[i]);
#pragma unroll
            for (int j = 0; j <= i; ++j) {
                kk[i][j] = fmaf(kv[i], kv[j], kk[i][j]);
                kq[i][j] = fmaf(qv[i], kv[j], kq[i][j]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < DELTA_BLOCK; ++i) {
        qq[i] = warp_sum(qq[i]);
#pragma unroll
        for (int j = 0; j <= i; ++j) {
            kk[i][j] = warp_sum(kk[i][j]);
            kq[i][j] = warp_sum(kq[i][j]);
        }
    }
    float k_inv[DELTA_BLOCK], q_inv[DELTA_BLOCK];
#pragma unroll
    for (int i = 0; i < DELTA_BLOCK; ++i) {
        k_inv[i] = 1.0f / sqrtf(kk[i][i] + DELTA_UNIT_EPS);
        q_inv[i] = s.q_scale / sqrtf(qq[i] + DELTA_UNIT_EPS);
    }
    // a lane per (head, token of the block)
    const int rep = s.H / s.G, me = lane & (DELTA_BLOCK - 1);
    for (int r0 = 0; r0 < rep; r0 += 32 / DELTA_BLOCK) {
        const int r = r0 + lane / DELTA_BLOCK, h = kvh * rep + min(r, rep - 1);
        float own = 0.f, beta = 0.f;
        if (me < n) delta_gates(z + (size_t)(t + me) * s.z_elems, s, h, decay[h], dt_bias[h], own, beta);
        float gm1[DELTA_BLOCK];              // g - 1 of every token of the block (0 beyond its end)
#pragma unroll
        for (int i = 0; i < DELTA_BLOCK; ++i) gm1[i] = __shfl_sync(0xffffffffu, own, i, DELTA_BLOCK);
        float till = 1.f, all = 0.f, Gm1 = 0.f;          // c_lj, G_l - 1, G_i - 1
#pragma unroll
        for (int i = 0; i < DELTA_BLOCK; ++i) {
            all = fmaf(all, gm1[i], all) + gm1[i];
            if (i == me) Gm1 = all;
            if (i > me) till = fmaf(till, gm1[i], till);
        }
        if (me >= n || r >= rep) continue;
        float4* dst = reinterpret_cast<float4*>(coef + ((size_t)(t + me) * s.H + h) * DELTA_COEF);
        const float G = 1.0f + Gm1;
#pragma unroll
        for (int i = 0; i < DELTA_BLOCK; ++i) {
            if (i != me) continue;
            float A[3] = {0.f, 0.f, 0.f}, B[DELTA_BLOCK] = {0.f, 0.f, 0.f, 0.f};
            float c = 1.f;                   // c_ij
#pragma unroll
            for (int j = i; j >= 0; --j) {
                B[j] = c * kq[i][j] * q_inv[i] * k_inv[j];
                if (j < i) A[j] = c * kk[i][j] * k_inv[i] * k_inv[j];
                c = fmaf(c, gm1[j], c);
            }
            dst[0] = make_float4(G * k_inv[i], beta, A[0], A[1]);
            dst[1] = make_float4(A[2], B[0], B[1], B[2]);
            dst[2] = make_float4(B[3], till * k_inv[i], G * q_inv[i], all);
        }
    }
}

// grid (sequences, heads, ceil(dv / (8 CPT))); 128 threads: thread = (group of CPT columns, ks), ks fastest.  Lane ks holds
// key channels ks * DPT .. ks * DPT + DPT - 1 of its columns (channels beyond d hold zeros).  A tile of tokens' q and k lie
// in shared memory as runs of DPT floats, each followed by 4 floats of padding, so that the lanes' 16-byte reads fall into
// different banks; the next tile's travel through registers meanwhile, as they are stored (a conversion would wait for
// them on the spot).  VEC: bfloat16 rows that allow loads of 8 channels.  Tokens beyond the sequence's end are zeros with
// G = 1, which change nothing.
template <typename T, int DPT, int CPT, bool VEC>
__global__ void __launch_bounds__(DELTA_NT, DPT <= 8 ? 4 : 1)
delta_scan_kernel(const T* __restrict__ x, DeltaShape s, const float* __restrict__ coef, const int* __restrict__ seq_slot,
                  const int* __restrict__ seq_first_row, const int* __restrict__ seq_start, const int* __restrict__ seq_end,
                  float* __restrict__ state, float* __restrict__ o_out) {
    constexpr int RUN = DPT + 4, TOK = DELTA_KS * RUN;
    constexpr int TT = DPT >= 16 ? 8 : 16;                     // tokens staged per round
    constexpr int COLS = DELTA_GROUPS * CPT, WIDTH = DELTA_KS * DPT, NB = DELTA_BLOCK;
    constexpr bool KEEP = DPT <= 8;                            // the block's keys stay in registers from the products to the update
    constexpr int PER = TT * WIDTH / DELTA_NT;
    constexpr int VPER = (TT * COLS + DELTA_NT - 1) / DELTA_NT, C4 = TT * DELTA_COEF / 4;
    static_assert(C4 <= DELTA_NT, "a thread carries one piece of the coefficients");
    __shared__ __align__(16) float q_s[TT * TOK];
    __shared__ __align__(16) float k_s[TT * TOK];
    __shared__ __align__(16) float c_s[TT * DELTA_COEF];
    __shared__ __align__(16) float v_s[TT * COLS];
    const int d = s.d, dv = s.dv, H = s.H;
    const int seq = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS, kvh = h / (H / s.G);
    const int tid = threadIdx.x, ks = tid % DELTA_KS, grp = tid / DELTA_KS, lane = tid & 31;
    grid_dependents_launch();
    const int slot = seq_slot[seq], row0 = seq_first_row[seq], n_tok = seq_end[seq] - seq_start[seq];
    if (n_tok <= 0) return;
    grid_dependency_wait();
    float S[CPT][DPT];
    float* st = slot >= 0 ? state + ((size_t)slot * H + h) * d * dv : nullptr;
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = col0 + grp * CPT + c;
#pragma unroll
        for (int ii = 0; ii < DPT; ++ii) {
            const int i = ks * DPT + ii;
            S[c][ii] = (st != nullptr && col < dv && i < d) ? st[(size_t)col * d + i] : 0.f;
        }
    }
    constexpr int PIECE = VEC ? 8 : 1, NP = PER / PIECE;
    typedef typename std::conditional<VEC, uint4, T>::type Raw;
    Raw qv[NP], kv[NP];
    T vv[VPER];
    const T zero = from_float<T>(0.f);
    float4 cf = make_float4(0.f, 0.f, 0.f, 0.f);
    auto fetch = [&](int t0) {
#pragma unroll
        for (int e = 0; e < NP; ++e) {
            const int u = (tid + e * DELTA_NT) * PIECE, tt = u / WIDTH, c = u % WIDTH;
            qv[e] = kv[e] = Raw{};
            if (t0 + tt < n_tok && c < d) {
                const T* row = x + (size_t)(row0 + t0 + tt) * s.x_elems + kvh * d + c;
                qv[e] = *reinterpret_cast<const Raw*>(row + s.q_off);
                kv[e] = *reinterpret_cast<const Raw*>(row + s.k_off);
            }
        }
#pragma unroll
        for (int e = 0; e < VPER; ++e) {
            const int u = tid + e * DELTA_NT, tt = u / COLS, c = col0 + u % COLS;
            vv[e] = zero;
            if (u < TT * COLS && t0 + tt < n_tok && c < dv) vv[e] = x[(size_t)(row0 + t0 + tt) * s.x_elems + s.v_off + h * dv + c];
        }
        if (tid < C4) {
            constexpr int P = DELTA_COEF / 4;
            const int tt = tid / P;
            cf = make_float4(0.f, 0.f, 0.f, 0.f);
            if (t0 + tt < n_tok)
                cf = reinterpret_cast<const float4*>(coef + ((size_t)(row0 + t0 + tt) * H + h) * DELTA_COEF)[tid % P];
        }
    };
    // one piece of a token's channels, from channel c on, into the token's runs
    auto put_piece = [](float* tok, int c, const Raw& raw) {
        if constexpr (VEC) {
            float f[8];
            Vec16<bf16>::load(reinterpret_cast<const bf16*>(&raw), f);
#pragma unroll
            for (int e = 0; e < 8; e += 4)
                *reinterpret_cast<float4*>(tok + ((c + e) / DPT) * RUN + (c + e) % DPT) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
        } else {
            tok[(c / DPT) * RUN + c % DPT] = to_float(raw);
        }
    };
    // which of a block's sums this lane ends up with: column, products with q (or with k), token
    const int my_c = CPT == 2 ? ks >> 3 : 0;
    const bool my_q = (CPT == 2 ? (ks >> 2) & 1 : ks >> 3) != 0;
    const int my_i = CPT == 2 ? ks & 3 : (ks >> 1) & 3;
    const int my_col = col0 + grp * CPT + my_c;
    const bool writer = my_q && my_col < dv && (CPT == 2 || (ks & 1) == 0);
    fetch(0);
    for (int t0 = 0; t0 < n_tok; t0 += TT) {
        __syncthreads();                       // the tile before has been read
#pragma unroll
        for (int e = 0; e < NP; ++e) {
            const int u = (tid + e * DELTA_NT) * PIECE, tt = u / WIDTH, c = u % WIDTH;
            put_piece(q_s + tt * TOK, c, qv[e]);
            put_piece(k_s + tt * TOK, c, kv[e]);
        }
#pragma unroll
        for (int e = 0; e < VPER; ++e)
            if (tid + e * DELTA_NT < TT * COLS) v_s[tid + e * DELTA_NT] = to_float(vv[e]);
        if (tid < C4) reinterpret_cast<float4*>(c_s)[tid] = cf;
        __syncthreads();
        if (t0 + TT < n_tok) fetch(t0 + TT);
#pragma unroll 1
        for (int b = 0; b < TT; b += NB) {
            if (t0 + b >= n_tok) break;
            // the block's products with the state before it
            float sum[8 * CPT];                // [column][k, q][token]
            float kr[KEEP ? NB : 1][DPT];      // this lane's run of the block's keys, for the update below
#pragma unroll
            for (int v = 0; v < 8 * CPT; ++v) sum[v] = 0.f;
#pragma unroll
            for (int i4 = 0; i4 < DPT / 4; ++i4) {
#pragma unroll
                for (int i = 0; i < NB; ++i) {
                    const float4 k4 = reinterpret_cast<const float4*>(k_s + (b + i) * TOK + ks * RUN)[i4];
                    const float4 q4 = reinterpret_cast<const float4*>(q_s + (b + i) * TOK + ks * RUN)[i4];
                    if (KEEP) {
                        float* k_ = &kr[KEEP ? i : 0][4 * i4];
                        k_[0] = k4.x; k_[1] = k4.y; k_[2] = k4.z; k_[3] = k4.w;
                    }
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        const float* Sc = &S[c][4 * i4];
                        float a = sum[c * 8 + i], o = sum[c * 8 + 4 + i];
                        a = fmaf(Sc[0], k4.x, a); a = fmaf(Sc[1], k4.y, a); a = fmaf(Sc[2], k4.z, a); a = fmaf(Sc[3], k4.w, a);
                        o = fmaf(Sc[0], q4.x, o); o = fmaf(Sc[1], q4.y, o); o = fmaf(Sc[2], q4.z, o); o = fmaf(Sc[3], q4.w, o);
                        sum[c * 8 + i] = a;
                        sum[c * 8 + 4 + i] = o;
                    }
                }
            }
            // the 16 lanes add their shares: every stage halves the sums a lane still carries (the lanes whose bit is set
            // keep the upper half)
            int n = 8 * CPT;
#pragma unroll
            for (int off = DELTA_KS / 2; off >= 1; off >>= 1) {
                const bool upper = (ks & off) != 0;
                if (n > 1) {
                    const int half = n / 2;
#pragma unroll
                    for (int i = 0; i < 4 * CPT; ++i)
                        if (i < half) {
                            const float mine = upper ? sum[i + half] : sum[i];
                            const float theirs = upper ? sum[i] : sum[i + half];
                            sum[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, off);
                        }
                    n = half;
                } else {
                    sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], off);
                }
            }
            const float mine = sum[0];
            // every lane solves for the block's u
            const float4* cb = reinterpret_cast<const float4*>(c_s + b * DELTA_COEF);
            float u[CPT][NB];
#pragma unroll
            for (int i = 0; i < NB; ++i) {
                const float4 c0 = cb[3 * i];
                const float A[3] = {c0.z, c0.w, i == 3 ? c_s[(b + i) * DELTA_COEF + 4] : 0.f};
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const float p = __shfl_sync(0xffffffffu, mine, (lane & 16) | (CPT == 2 ? c * 8 + i : 2 * i));
                    float r = fmaf(-c0.x, p, v_s[(b + i) * COLS + grp * CPT + c]);
#pragma unroll
                    for (int j = 0; j < i; ++j) r = fmaf(-A[j], u[c][j], r);
                    u[c][i] = c0.y * r;
                }
            }
            if (writer && t0 + b + my_i < n_tok) {
                const float* ci = c_s + (b + my_i) * DELTA_COEF;
                float o = ci[10] * mine;
#pragma unroll
                for (int j = 0; j < NB; ++j) o = fmaf(ci[5 + j], CPT == 2 && my_c ? u[CPT - 1][j] : u[0][j], o);
                o_out[(size_t)(row0 + t0 + b + my_i) * H * dv + h * dv + my_col] = o;
            }
            float gm1 = 0.f;
#pragma unroll
            for (int j = 0; j < NB; ++j) {
                const float4 c2 = cb[3 * j + 2];
                if (j == 0) gm1 = c2.w;
#pragma unroll
                for (int c = 0; c < CPT; ++c) u[c][j] *= c2.y;
            }
#pragma unroll
            for (int i4 = 0; i4 < DPT / 4; ++i4) {
                float add[CPT][4];
#pragma unroll
                for (int c = 0; c < CPT; ++c)
#pragma unroll
                    for (int e = 0; e < 4; ++e) add[c][e] = S[c][4 * i4 + e] * gm1;
#pragma unroll
                for (int j = 0; j < NB; ++j) {
                    float k_[4];
                    if (KEEP) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) k_[e] = kr[KEEP ? j : 0][4 * i4 + e];
                    } else {
                        const float4 k4 = reinterpret_cast<const float4*>(k_s + (b + j) * TOK + ks * RUN)[i4];
                        k_[0] = k4.x; k_[1] = k4.y; k_[2] = k4.z; k_[3] = k4.w;
                    }
#pragma unroll
                    for (int c = 0; c < CPT; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) add[c][e] = fmaf(k_[e], u[c][j], add[c][e]);
                }
#pragma unroll
                for (int c = 0; c < CPT; ++c)
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[c][4 * i4 + e] += add[c][e];
            }
        }
    }
    if (st != nullptr) {
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int col = col0 + grp * CPT + c;
#pragma unroll
            for (int ii = 0; ii < DPT; ++ii) {
                const int i = ks * DPT + ii;
                if (col < dv && i < d) st[(size_t)col * d + i] = S[c][ii];
            }
        }
    }
}

// Steps of single rows (decoding): the recurrence, the norm of the head's output and its gate in one launch.  A CTA per
// (head, sequence), LANES lanes a column of the state, JN pieces of VEC channels a lane; a warp takes several columns at
// once, so that many of their loads are on their way together.  Both products are with the state as it was stored,
//   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T
// and the state is read and written once.
constexpr int DELTA_STEP_WARPS = 8;

struct DeltaGate {
    int g_off;                    // the gate's logits [H, dv] in a projected row
    float eps;
    const float* w;               // [dv]
};

template <typename T, int LANES, int VEC, int JN>
__global__ void __launch_bounds__(DELTA_STEP_WARPS * 32)
delta_step_kernel(const T* __restrict__ x, const T* __restrict__ z, DeltaShape s, const float* __restrict__ decay,
                  const float* __restrict__ dt_bias, const int* __restrict__ tok_seq, const int* __restrict__ seq_slot,
                  float* __restrict__ state, DeltaGate gate, T* __restrict__ out) {
    constexpr int PAR = 32 / LANES, AT_ONCE = JN * VEC <= 4 ? 8 : (JN * VEC <= 8 ? 4 : 2);     // columns a warp, a lane in flight
    extern __shared__ float o_s[];                  // [dv]
    __shared__ float scratch[32];
    const int h = blockIdx.x, t = blockIdx.y, d = s.d, dv = s.dv, kvh = h / (s.H / s.G);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, li = lane % LANES, sub = lane / LANES;
    grid_dependents_launch();
    const int slot = seq_slot[tok_seq[t]];
    const float dec = decay[h], dtb = dt_bias[h];
    grid_dependency_wait();
    const T* xr = x + (size_t)t * s.x_elems;
    const T* zr = z + (size_t)t * s.z_elems;
    float k[JN][VEC], q[JN][VEC], kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
    for (int j = 0; j < JN; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const int i = (j * LANES + li) * VEC + e;
            k[j][e] = i < d ? to_float(xr[s.k_off + kvh * d + i]) : 0.f;
            q[j][e] = i < d ? to_float(xr[s.q_off + kvh * d + i]) : 0.f;
            kk = fmaf(k[j][e], k[j][e], kk);
            qq = fmaf(q[j][e], q[j][e], qq);
            kq = fmaf(k[j][e], q[j][e], kq);
        }
    float gm1, beta;
    delta_gates(zr, s, h, dec, dtb, gm1, beta);
    auto lanes_sum = [](float v) {
#pragma unroll
        for (int off = LANES / 2; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
        return v;
    };
    kk = lanes_sum(kk);
    qq = lanes_sum(qq);
    kq = lanes_sum(kq);
    const float k_inv = 1.0f / sqrtf(kk + DELTA_UNIT_EPS), q_inv = s.q_scale / sqrtf(qq + DELTA_UNIT_EPS), g = 1.0f + gm1;
    kq *= k_inv * q_inv;
#pragma unroll
    for (int j = 0; j < JN; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            k[j][e] *= k_inv;
            q[j][e] *= q_inv;
        }
    float* st = slot >= 0 ? state + ((size_t)slot * s.H + h) * d * dv : nullptr;
    constexpr int STEP = DELTA_STEP_WARPS * PAR;
    for (int c0 = warp * PAR + sub; c0 - sub < dv; c0 += STEP * AT_ONCE) {
        float S[AT_ONCE][JN][VEC], v[AT_ONCE];
#pragma unroll
        for (int a = 0; a < AT_ONCE; ++a) {
            const int col = c0 + a * STEP;
            v[a] = col < dv ? to_float(xr[s.v_off + h * dv + col]) : 0.f;
#pragma unroll
            for (int j = 0; j < JN; ++j) {
                const int i = (j * LANES + li) * VEC;
#pragma unroll
                for (int e = 0; e < VEC; ++e) S[a][j][e] = 0.f;
                if (st != nullptr && col < dv && i < d) {
                    if (VEC == 4) {
                        const float4 s4 = *reinterpret_cast<const float4*>(st + (size_t)col * d + i);
                        S[a][j][0] = s4.x; S[a][j][VEC > 1 ? 1 : 0] = s4.y; S[a][j][VEC > 2 ? 2 : 0] = s4.z; S[a][j][VEC > 3 ? 3 : 0] = s4.w;
                    } else {
                        S[a][j][0] = st[(size_t)col * d + i];
                    }
                }
            }
        }
#pragma unroll
        for (int a = 0; a < AT_ONCE; ++a) {
            const int col = c0 + a * STEP;
            float pk = 0.f, pq = 0.f;
#pragma unroll
            for (int j = 0; j < JN; ++j)
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    pk = fmaf(S[a][j][e], k[j][e], pk);
                    pq = fmaf(S[a][j][e], q[j][e], pq);
                }
            pk = lanes_sum(pk);
            pq = lanes_sum(pq);
            const float u = beta * fmaf(-g, pk, v[a]);
            if (li == 0 && col < dv) o_s[col] = fmaf(kq, u, g * pq);
            if (st != nullptr && col < dv) {
#pragma unroll
                for (int j = 0; j < JN; ++j) {
                    const int i = (j * LANES + li) * VEC;
                    if (i >= d) continue;
#pragma unroll
                    for (int e = 0; e < VEC; ++e) S[a][j][e] += fmaf(k[j][e], u, S[a][j][e] * gm1);
                    if (VEC == 4)
                        *reinterpret_cast<float4*>(st + (size_t)col * d + i) =
                            make_float4(S[a][j][0], S[a][j][VEC > 1 ? 1 : 0], S[a][j][VEC > 2 ? 2 : 0], S[a][j][VEC > 3 ? 3 : 0]);
                    else
                        st[(size_t)col * d + i] = S[a][j][0];
                }
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) ss = fmaf(o_s[c], o_s[c], ss);
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)dv + gate.eps);
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        const float gv = to_float(zr[gate.g_off + h * dv + c]);
        out[((size_t)t * s.H + h) * dv + c] = from_float<T>(o_s[c] * inv * gate.w[c] * (gv / (1.0f + expf(-gv))));
    }
}

}  // namespace janis

using namespace janis;

static int delta_check(const char* what, const DeltaShape& s) {
    if (s.H <= 0 || s.G <= 0 || s.H % s.G || s.d <= 0 || s.dv <= 0) return fail("%s: sizes %d heads over %d, %d x %d", what, s.H, s.G, s.d, s.dv);
    if (s.d > DELTA_KS * 16) return fail("%s: key size %d is above %d", what, s.d, DELTA_KS * 16);
    if (s.H > 65535) return fail("%s: too many heads (%d)", what, s.H);
    if (s.q_off < 0 || s.k_off < 0 || s.v_off < 0 || s.q_off + s.G * s.d > s.x_elems || s.k_off + s.G * s.d > s.x_elems ||
        s.v_off + s.H * s.dv > s.x_elems)
        return fail("%s: queries, keys and values do not fit rows of %d", what, s.x_elems);
    if (s.a_off < 0 || s.b_off < 0 || s.a_off + s.H > s.z_elems || s.b_off + s.H > s.z_elems)
        return fail("%s: the gates do not fit rows of %d", what, s.z_elems);
    return 0;
}

template <typename T>
static int delta_prompt_launch(const void* x, const void* z, const DeltaShape& s, const float* decay, const float* dt_bias, float* coef,
                               const int* tok_pos, const int* tok_seq, const int* seq_slot, const int* seq_first_row,
                               const int* seq_start, const int* seq_end, float* state, float* o_out, int n_seq, int n_tok,
                               int form, cudaStream_t stream) {
    const int warps = s.G < 4 ? s.G : 4;
    if (launch_kernel("delta_coef", delta_coef_kernel<T>, dim3(n_tok, (s.G + warps - 1) / warps), dim3(warps * 32), 0, stream, 1, (const T*)x,
                      (const T*)z, s, decay, dt_bias, tok_pos, tok_seq, seq_start, seq_end, coef, n_tok))
        return 1;
    // two columns a group of lanes halve the reads from shared memory and the exchanges a column; where one column a group
    // leaves every CTA an SM of its own that is faster still
    const bool two = form ? form == 2 : (long long)n_seq * s.H * ((s.dv + DELTA_GROUPS - 1) / DELTA_GROUPS) > 148;
    const int cols = DELTA_GROUPS * (two ? 2 : 1);
    const dim3 grid(n_seq, s.H, (s.dv + cols - 1) / cols), block(DELTA_NT);
    // 16-byte loads (8 channels of one token a piece) where the rows allow it, else element by element
    const bool vec = sizeof(T) == 2 && s.d % 8 == 0 && s.x_elems % 8 == 0 && s.q_off % 8 == 0 && s.k_off % 8 == 0 && ((uintptr_t)x & 15) == 0;
#define JANIS_DELTA_LAUNCH(DPT, CPT)                                                                                   \
    return launch_kernel_after("delta_scan", vec ? delta_scan_kernel<T, DPT, CPT, sizeof(T) == 2> : delta_scan_kernel<T, DPT, CPT, false>, grid, block, 0, stream, 1, (const T*)x, s, (const float*)coef, \
                         seq_slot, seq_first_row, seq_start, seq_end, state, o_out);
#define JANIS_DELTA_CASE(DPT)                                                                                          \
    if (s.d <= DELTA_KS * DPT) {                                                                                       \
        if (two) { JANIS_DELTA_LAUNCH(DPT, 2) }                                                                   \
        JANIS_DELTA_LAUNCH(DPT, 1)                                                                                     \
    }
    JANIS_DELTA_CASE(4)
    JANIS_DELTA_CASE(8)
    JANIS_DELTA_CASE(16)
#undef JANIS_DELTA_CASE
#undef JANIS_DELTA_LAUNCH
    return fail("delta_scan: key size %d is above %d", s.d, DELTA_KS * 16);
}

// x: the convolved rows [n_tok, x_elems] (q [G, d], k [G, d], v [H, dv] at their offsets); z: the projected rows (za [H] at
// a_off, zb [H] at b_off); decay, dt_bias [H] float; coef: float scratch [n_tok, H, 12]; state float [slots, H, dv, d];
// o_out float [n_tok, H dv].  form: 1 or 2 fixes the columns a group of lanes takes (0: chosen from the step's size).
JANIS_EXPORT int janis_delta_scan(const void* x, int x_elems, int q_off, int k_off, int v_off, const void* z, int z_elems, int a_off,
                                  int b_off, int dtype, const float* decay, const float* dt_bias, float q_scale, float* coef,
                                  const int* tok_pos, const int* tok_seq, const int* seq_slot, const int* seq_first_row,
                                  const int* seq_start, const int* seq_end, float* state, float* o_out, int n_seq, int n_tok,
                                  int H, int G, int d, int dv, int form, cudaStream_t stream) {
    if (n_seq <= 0 || n_tok <= 0) return 0;
    const DeltaShape s = {H, G, d, dv, x_elems, q_off, k_off, v_off, z_elems, a_off, b_off, q_scale};
    if (delta_check("delta_scan", s)) return 1;
    if (form < 0 || form > 2) return fail("delta_scan: %d columns a group of lanes", form);
    if (((uintptr_t)coef) & 15) return fail("delta_scan: the coefficients start on a 16-byte border");
    if (dtype == JANIS_F32)
        return delta_prompt_launch<float>(x, z, s, decay, dt_bias, coef, tok_pos, tok_seq, seq_slot, seq_first_row, seq_start, seq_end,
                                          state, o_out, n_seq, n_tok, form, stream);
    if (dtype == JANIS_BF16)
        return delta_prompt_launch<bf16>(x, z, s, decay, dt_bias, coef, tok_pos, tok_seq, seq_slot, seq_first_row, seq_start, seq_end,
                                         state, o_out, n_seq, n_tok, form, stream);
    return fail("delta_scan: unknown dtype %d", dtype);
}

template <typename T>
static int delta_step_launch(const void* x, const void* z, const DeltaShape& s, const float* decay, const float* dt_bias,
                             const int* tok_seq, const int* seq_slot, float* state, const DeltaGate& g, void* out, int n_rows,
                             cudaStream_t stream) {
    const dim3 grid(s.H, n_rows), block(DELTA_STEP_WARPS * 32);
    const size_t bytes = (size_t)s.dv * sizeof(float);
#define JANIS_DELTA_STEP(LANES, VEC, JN)                                                                               \
    return launch_kernel("delta_step", delta_step_kernel<T, LANES, VEC, JN>, grid, block, bytes, stream, 1, (const T*)x, \
                         (const T*)z, s, decay, dt_bias, tok_seq, seq_slot, state, g, (T*)out);
    if (s.d % 4 == 0 && ((uintptr_t)state & 15) == 0) {
        if (s.d <= 32) { JANIS_DELTA_STEP(8, 4, 1) }
        if (s.d <= 64) { JANIS_DELTA_STEP(16, 4, 1) }
        if (s.d <= 128) { JANIS_DELTA_STEP(32, 4, 1) }
        JANIS_DELTA_STEP(32, 4, 2)
    }
    if (s.d <= 64) { JANIS_DELTA_STEP(32, 1, 2) }
    JANIS_DELTA_STEP(32, 1, 8)
#undef JANIS_DELTA_STEP
}

// One token a row: x, z, decay, dt_bias and state as above; the gate's logits [H, dv] at g_off of z; norm_w [dv]; out
// [n_rows, H dv] in the activation type: the head's output over its root mean square, times norm_w, times silu(gate).
JANIS_EXPORT int janis_delta_step(const void* x, int x_elems, int q_off, int k_off, int v_off, const void* z, int z_elems, int a_off,
                                  int b_off, int g_off, int dtype, const float* decay, const float* dt_bias, float q_scale,
                                  const float* norm_w, float eps, const int* tok_seq, const int* seq_slot, float* state, void* out,
                                  int n_rows, int H, int G, int d, int dv, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    const DeltaShape s = {H, G, d, dv, x_elems, q_off, k_off, v_off, z_elems, a_off, b_off, q_scale};
    if (delta_check("delta_step", s)) return 1;
    if (g_off < 0 || g_off + H * dv > z_elems) return fail("delta_step: the gate does not fit rows of %d", z_elems);
    if (n_rows > 65535) return fail("delta_step: %d rows", n_rows);
    if (dv > 8192) return fail("delta_step: a head of %d values", dv);
    const DeltaGate g = {g_off, eps, norm_w};
    if (dtype == JANIS_F32) return delta_step_launch<float>(x, z, s, decay, dt_bias, tok_seq, seq_slot, state, g, out, n_rows, stream);
    if (dtype == JANIS_BF16) return delta_step_launch<bf16>(x, z, s, decay, dt_bias, tok_seq, seq_slot, state, g, out, n_rows, stream);
    return fail("delta_step: unknown dtype %d", dtype);
}
