// Recurrences whose state per head is a matrix: S_t = a_t S_{t-1} + b_t k_t v_t^T,
// y_t = S_t^T q_t + d v_t, with S of N x P values per head in float32, carried from step
// to step per slot.  Two mixers are instances of it:
//
//   selective state space (Mamba-2's form): per head h of H, with group g = h / (H / G)
//       dt = softplus(dt_sum + dt_bias_h);  a = exp(-exp(A_log_h) dt);  b = dt
//       k = B_g, q = C_g (N values), v = x_h (P values), d = D_h
//   linear attention with a decay per head: a = decay_h, b = 1, d = 0, k, q, v the silu of
//       the products' sums, G = H
//   matrix memory with exponential gates (mLSTM): log gates i = c(zi), f = log sigmoid(c(zf)), c(z) =
//       cap tanh(z / cap), a running maximum m_t = max(f + m_{t-1}, i), a = e^(f + m_{t-1} - m_t),
//       b = e^(i - m_t), d = 0, G = H, and beside S a vector n_t = a n_{t-1} + b k_t per head, whose
//       product with q divides y: y / (max(|n . q|, e^(-m_t)) + floor)
//
// and what follows them: a gate and an RMS norm in equal parts of the row, and the sum of
// two mixers' results.  Everything here is float32: steps, decays, exponentials, the
// state, the norms.
//
// Rows are the sequences' tokens one sequence after the other (row_seq is sorted), so a
// sequence's rows are found by a search in row_seq; nothing comes from the host, and a
// captured decode step replays with other contents.
#include "common.cuh"
#include "kernels.h"

namespace jb {

// The sums of a gated memory's two log gates: H columns each of [S, n, ld], biases [H], the soft cap.
struct LogGates {
    const float *src;
    int S;
    size_t stride;
    int ld, i_col0, f_col0;
    const float *i_bias, *f_bias;
    float cap;
};

struct ScanIn {
    const float *src;          // sums [S, n, ld] that hold v, k and q
    int S;
    size_t stride;
    int ld, val_col0, key_col0, qry_col0;
    int silu;                  // v, k, q are silu(sum)
    const float *dt;           // sums [dt_S, n, dt_ld] with the steps' columns, or null
    int dt_S;
    size_t dt_stride;
    int dt_ld, dt_col0;
    const float *dt_bias, *a_log, *skip;      // [H] each (with dt)
    const float *decay;                       // [H] (without dt)
    // exponential gates (GATED kernels): per row and head a and b as they are ([n, H] each), or with
    // coef_a null from the gates' sums and the running maximum in the state (a decode step's rows)
    const float *coef_a, *coef_b;
    LogGates gates;
    float q_scale;             // y and nq are multiplied by it
    float *nq;                 // [n, H]: n . q
};

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
// log(1 + e^v), the same number as the direct form wherever that does not overflow
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// row r's sums of the two log gates of head h, and the gates from them
__device__ __forceinline__ void gate_sums(const LogGates &g, int r, int h, float &zi, float &zf)
{
    const float *row = g.src + (size_t)r * g.ld + h;
    zi = add_partials(g.i_bias[h], row + g.i_col0, g.S, g.stride);
    zf = add_partials(g.f_bias[h], row + g.f_col0, g.S, g.stride);
}
__device__ __forceinline__ void gates_of(float cap, float zi, float zf, float &i, float &f)
{
    i = cap * tanhf(zi / cap);
    zf = cap * tanhf(zf / cap);
    f = fminf(zf, 0.0f) - log1pf(expf(-fabsf(zf)));
}
__device__ __forceinline__ void log_gates(const LogGates &g, int r, int h, float &i, float &f)
{
    float zi, zf;
    gate_sums(g, r, h, zi, zf);
    gates_of(g.cap, zi, zf, i, f);
}

// an asynchronous copy of BYTES (4 or 16) from global to shared memory, and the wait for all of a thread's
template <int BYTES>
__device__ __forceinline__ void copy_async(float *smem, const float *gmem)
{
    uint32_t dst = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(dst), "l"(gmem), "n"(BYTES) : "memory");
}
__device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// first row r with row_seq[r] >= s
__device__ __forceinline__ int first_row_of(const int32_t *__restrict__ row_seq, int n, int s)
{
    int lo = 0, hi = n;
    while (lo < hi) {
        int mid = (lo + hi) >> 1;
        if (row_seq[mid] < s)
            lo = mid + 1;
        else
            hi = mid;
    }
    return lo;
}

// The gates of a step's rows ahead of a prompt's recurrence: a, b and e^(-m) per row and head, and the
// slots' running maximum after the step (at m_off + h of a slot's state).  A block per (head,
// sequence); a thread has consecutive rows, whose maps m -> max(m + F, M) are composed across the
// block to give every thread the maximum it starts from.  HELD: the most rows a thread keeps the gates
// of (0: any number, their sums are read and their gates taken twice).
constexpr int LG_THREADS = 512;
template <int HELD>
__global__ void __launch_bounds__(LG_THREADS)
log_gates_kernel(LogGates g, float *__restrict__ state, size_t slot_stride, size_t m_off,
                 const int32_t *__restrict__ row_seq, const int32_t *__restrict__ seq_slot,
                 float *__restrict__ coef_a, float *__restrict__ coef_b, float *__restrict__ em, int n, int H)
{
    __shared__ float wF[LG_THREADS / 32], wM[LG_THREADS / 32], last[LG_THREADS];
    pdl_trigger();
    int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int r0 = first_row_of(row_seq, n, seq), r1 = first_row_of(row_seq, n, seq + 1);
    if (r0 >= r1)
        return;
    int per = (r1 - r0 + LG_THREADS - 1) / LG_THREADS;
    int t0 = min(r1, r0 + tid * per), t1 = min(r1, t0 + per);
    float *mp = state + (size_t)seq_slot[seq] * slot_stride + m_off + h;
    pdl_wait();
    float m0 = *mp, F = 0.0f, M = -INFINITY;
    constexpr int CAP = HELD > 0 ? HELD : 1;
    float gi[CAP], gf[CAP];
    if (HELD > 0) {
        // (rows past the thread's last repeat it: the loads go out together)
#pragma unroll
        for (int k = 0; k < CAP; k++)
            gate_sums(g, min(t0 + k, r1 - 1), h, gi[k], gf[k]);
#pragma unroll
        for (int k = 0; k < CAP; k++)
            gates_of(g.cap, gi[k], gf[k], gi[k], gf[k]);
#pragma unroll
        for (int k = 0; k < CAP; k++)
            if (t0 + k < t1) {
                F += gf[k];
                M = fmaxf(M + gf[k], gi[k]);
            }
    } else {
        for (int r = t0; r < t1; r++) {
            float i, f;
            log_gates(g, r, h, i, f);
            F += f;
            M = fmaxf(M + f, i);
        }
    }
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
        float eF = __shfl_up_sync(0xffffffffu, F, o), eM = __shfl_up_sync(0xffffffffu, M, o);
        if (lane >= o) {
            M = fmaxf(eM + F, M);
            F += eF;
        }
    }
    if (lane == 31) {
        wF[warp] = F;
        wM[warp] = M;
    }
    F = __shfl_up_sync(0xffffffffu, F, 1);
    M = __shfl_up_sync(0xffffffffu, M, 1);
    __syncthreads();
    float m = m0;
    for (int w = 0; w < warp; w++)
        m = fmaxf(m + wF[w], wM[w]);
    if (lane > 0)
        m = fmaxf(m + F, M);
    // The first row's a is taken from the maximum that the thread before arrived at, not from the
    // composed one, which differs from it in rounding: the products of the a telescope exactly.
    float first_f = 0.0f, first_m = 0.0f;
    auto row = [&](int r, float i, float f) {
        float mn = fmaxf(f + m, i);
        if (r == t0) {
            first_f = f;
            first_m = mn;
        } else {
            coef_a[(size_t)r * H + h] = expf(f + m - mn);
        }
        coef_b[(size_t)r * H + h] = expf(i - mn);
        em[(size_t)r * H + h] = expf(-mn);
        m = mn;
    };
    if (HELD > 0) {
#pragma unroll
        for (int k = 0; k < CAP; k++)
            if (t0 + k < t1)
                row(t0 + k, gi[k], gf[k]);
    } else {
        for (int r = t0; r < t1; r++) {
            float i, f;
            log_gates(g, r, h, i, f);
            row(r, i, f);
        }
    }
    last[tid] = m;
    __syncthreads();
    if (t0 < t1) {
        float before = tid > 0 ? last[tid - 1] : m0;
        coef_a[(size_t)t0 * H + h] = expf(first_f + before - first_m);
        if (t1 == r1)
            *mp = m;
    }
}

// The vector n of a gated memory over rows r0 .. r1 - 1 of one head: n <- a n + b k, and n . q
// times q_scale to in.nq (MODE as in the kernel below: MODE 1 gives no n . q).  128 threads, one value
// each, 128 values of n after the others.  from null: zeros; to null: nothing is written back.
template <int MODE>
__device__ __forceinline__ void normaliser_rows(const ScanIn &in, const float *from, float *to, int r0, int r1,
                                                int H, int h, int N, float m_before, float (*red)[8])
{
    constexpr int TB = 8;
    int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    auto sum = [&in](const float *p) {
        float v = p[0];
#pragma unroll 1
        for (int k = 1; k < in.S; k++)
            v += p[(size_t)k * in.stride];
        return v;
    };
#pragma unroll 1
    for (int n0 = 0; n0 < N; n0 += 128) {
        bool live = n0 + tid < N;
        float nv = from != nullptr && live ? from[n0 + tid] : 0.0f;
        const float *col = in.src + (size_t)h * N + n0 + tid;
#pragma unroll 1
        for (int c0 = r0; c0 < r1; c0 += TB) {
            int tb = min(TB, r1 - c0);
            float k[TB], part[TB], a[TB], b[TB];
#pragma unroll
            for (int tt = 0; tt < TB; tt++) {
                int r = min(c0 + tt, r1 - 1);
                const float *row = col + (size_t)r * in.ld;
                k[tt] = live ? sum(row + in.key_col0) : 0.0f;
                part[tt] = MODE != 1 && live ? sum(row + in.qry_col0) : 0.0f;
                if (in.coef_a != nullptr) {
                    a[tt] = in.coef_a[(size_t)r * H + h];
                    b[tt] = in.coef_b[(size_t)r * H + h];
                }
            }
            if (in.coef_a == nullptr) {          // a decode step: one row
                float i, f;
                log_gates(in.gates, c0, h, i, f);
                float mn = fmaxf(f + m_before, i);
                a[0] = expf(f + m_before - mn);
                b[0] = expf(i - mn);
            }
#pragma unroll
            for (int tt = 0; tt < TB; tt++)
                if (tt < tb) {
                    nv = fmaf(b[tt], k[tt], a[tt] * nv);
                    part[tt] *= nv;
                }
            if (MODE != 1) {
#pragma unroll
                for (int tt = 0; tt < TB; tt++) {
                    part[tt] = warp_sum(part[tt]);
                    if (lane == 0)
                        red[warp][tt] = part[tt];
                }
                __syncthreads();
                if (tid < tb) {
                    float *o = in.nq + (size_t)(c0 + tid) * H + h;
                    float v = ((red[0][tid] + red[1][tid]) + (red[2][tid] + red[3][tid])) * in.q_scale;
                    *o = n0 > 0 ? *o + v : v;
                }
                __syncthreads();
            }
        }
        if (to != nullptr && live)
            to[n0 + tid] = nv;
    }
}

// A block of 128 threads per (tile of P, head, sequence or piece of one).  A warp has
// PW = 32 / nsplit columns p of the state, consecutive in memory, and nsplit lanes to a column;
// the lanes of a column hold the rows n = (i nsplit + ns) 4 + j of it in registers (up to NR),
// so that four rows' k and q come from shared memory in one load that the lanes of a column
// share out among them.  The block walks its rows in order, TB rows' k, q, v, a and b brought
// into shared memory together (by asynchronous copies where the sums are the values themselves);
// the lanes of a column add their parts of y with shuffles.
//
// MODE 0: a sequence's rows of the step from the slot's state; y and the state are written.
// MODE 1: a piece of `piece` rows from a state of zeros: the piece's own end state goes to
//         local[z] and the product of its decays to decays[z, h] (no y).
// MODE 2: a piece from the state in local[z] (what carry_kernel left there); y is written, and
//         by a sequence's last piece the slot's state.
// With pieces, blockIdx.z counts (sequence, piece); pieces that hold no row return.
// (local is no __restrict__ argument: MODE 2 only reads it, and the compiler might then fetch it ahead
// of pdl_wait.)
// NS: the split where it is fixed at compile time (0: nsplit_arg says it).
// GATED: exponential gates.  The state per head is then [N P | N] with n behind S, all heads' running
// maxima follow ([H]), and one block more along x walks n.  The running maximum is not written here.
// state: [H, N, P] per slot, slot_stride floats apart.  y: float32 [n, H P].
template <int NR, int TB, int MODE, int NS, bool GATED>
__global__ void __launch_bounds__(128, NR <= 16 ? 5 : 3)
matrix_state_scan_kernel(ScanIn in, float *__restrict__ state, size_t slot_stride,
                         const int32_t *__restrict__ row_seq, const int32_t *__restrict__ seq_slot,
                         float *__restrict__ y, float *local, float *decays, int n,
                         int H, int G, int N, int P, int nsplit_arg, int every_row_starts, int piece, int pieces)
{
    extern __shared__ float4 sm4[];
    float *sm = reinterpret_cast<float *>(sm4);
    pdl_trigger();
    // NS > 0: the split is known when the kernel is compiled and every lane has exactly NR rows
    // (N = NR NS), so that the places in shared memory are constants and no row needs a check
    const int nsplit = NS > 0 ? NS : nsplit_arg;
    const int PW = 32 / nsplit, PT = 4 * PW;
    const int NP = NS > 0 ? NR * NS : (N + 4 * nsplit - 1) / (4 * nsplit) * (4 * nsplit);   // rows, padded with zeros
    const int cnt4 = NS > 0 ? NR / 4 : NP / (4 * nsplit);                    // groups of four rows a lane
    int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int ns = lane / PW, pl = warp * PW + lane % PW;
    int p = blockIdx.x * PT + pl, h = blockIdx.y;
    int seq = MODE == 0 ? blockIdx.z : blockIdx.z / pieces, pc = MODE == 0 ? 0 : blockIdx.z % pieces;
    int g = h / (H / G);
    float *key_s = sm, *qry_s = key_s + TB * NP, *val_s = qry_s + (MODE == 1 ? 0 : TB * NP), *a_s = val_s + TB * PT,
          *b_s = a_s + TB;
    int r0, r1;
    if (every_row_starts) {
        r0 = seq;
        r1 = seq + 1;
    } else {
        r0 = first_row_of(row_seq, n, seq);
        r1 = first_row_of(row_seq, n, seq + 1);
    }
    bool last_piece = true;
    if (MODE != 0) {
        // A sequence that brings fewer than two pieces' rows stays whole (its first piece has
        // all its rows), so that its sums are added in the order of the one-pass form: what
        // else the step holds then does not change a sequence's bits.
        int end = r1;
        if (r1 - r0 >= 2 * piece) {
            r0 += pc * piece;
            r1 = min(r1, r0 + piece);
        } else if (pc > 0) {
            return;
        }
        last_piece = r1 == end;
    }
    if (r0 >= r1)
        return;
    const size_t per_head = (size_t)N * P + (GATED ? N : 0);
    float *slot = state + (size_t)seq_slot[seq] * slot_stride;
    float *st = MODE == 0 ? slot + (size_t)h * per_head : local + ((size_t)blockIdx.z * H + h) * per_head;
    bool live = p < P;
    float dskip = !GATED && in.dt != nullptr && in.skip != nullptr ? in.skip[h] : 0.0f;
    float a_neg = !GATED && in.dt != nullptr ? -expf(in.a_log[h]) : 0.0f;
    pdl_wait();
    float m_before = GATED && in.coef_a == nullptr ? slot[(size_t)H * per_head + h] : 0.0f;
    if (GATED && blockIdx.x == gridDim.x - 1) {
        __shared__ float red[4][8];
        const float *from = MODE == 1 ? nullptr : st + (size_t)N * P;
        float *to = MODE != 2 ? st + (size_t)N * P
                              : last_piece ? slot + (size_t)h * per_head + (size_t)N * P : nullptr;
        normaliser_rows<MODE>(in, from, to, r0, r1, H, h, N, m_before, red);
        return;
    }
    float s[NR];
#pragma unroll
    for (int i = 0; i < NR; i++) {
        int nn = ((i >> 2) * nsplit + ns) * 4 + (i & 3);
        s[i] = MODE != 1 && live && nn < N ? st[(size_t)nn * P + p] : 0.0f;
    }
    float run = 1.0f;        // the product of the piece's decays
    // TB rows' k, q, v, a and b at a time.  Where the sums are the values themselves (one partial
    // sum, no activation) they go from memory into shared memory by asynchronous copies, all of a
    // batch in flight together, 16 bytes each where everything lies on such boundaries; otherwise
    // the threads add and activate them on the way.
    const bool direct = in.S == 1 && !in.silu;
    const float *__restrict__ src = in.src;
    const int kcol = in.key_col0 + g * N, qcol = in.qry_col0 + g * N, vcol = in.val_col0 + h * P + blockIdx.x * PT;
    const bool k16 = direct && N % 4 == 0 && in.ld % 4 == 0 && kcol % 4 == 0 && qcol % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(src) & 15) == 0;
    const bool v16 = direct && PT % 4 == 0 && P % 4 == 0 && in.ld % 4 == 0 && vcol % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(src) & 15) == 0;
    if (direct) {
        // the rows' padding beyond N is never copied over: zeros once
        for (int i = tid; i < TB * (NP - N); i += 128) {
            int tt = i / (NP - N), nn = N + i - tt * (NP - N);
            key_s[tt * NP + nn] = 0.0f;
            if (MODE != 1)
                qry_s[tt * NP + nn] = 0.0f;
        }
    }
    for (int c0 = r0; c0 < r1; c0 += TB) {
        int tb = min(TB, r1 - c0);
        __syncthreads();
        if (direct) {
            if (k16) {
                int n4 = N / 4;
                for (int i = tid; i < tb * n4; i += 128) {
                    int tt = i / n4, c4 = (i - tt * n4) * 4;
                    const float *row = src + (size_t)(c0 + tt) * in.ld + c4;
                    copy_async<16>(key_s + tt * NP + c4, row + kcol);
                    if (MODE != 1)
                        copy_async<16>(qry_s + tt * NP + c4, row + qcol);
                }
            } else {
                for (int i = tid; i < tb * N; i += 128) {
                    int tt = i / N, nn = i - tt * N;
                    const float *row = src + (size_t)(c0 + tt) * in.ld + nn;
                    copy_async<4>(key_s + tt * NP + nn, row + kcol);
                    if (MODE != 1)
                        copy_async<4>(qry_s + tt * NP + nn, row + qcol);
                }
            }
            if (v16) {
                int p4 = PT / 4;
                for (int i = tid; i < tb * p4; i += 128) {
                    int tt = i / p4, c4 = (i - tt * p4) * 4;
                    if (blockIdx.x * PT + c4 < P)
                        copy_async<16>(val_s + tt * PT + c4, src + (size_t)(c0 + tt) * in.ld + vcol + c4);
                    else
                        *reinterpret_cast<float4 *>(val_s + tt * PT + c4) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                }
            } else {
                for (int i = tid; i < tb * PT; i += 128) {
                    int tt = i / PT, pp = i - tt * PT;
                    if (blockIdx.x * PT + pp < P)
                        copy_async<4>(val_s + i, src + (size_t)(c0 + tt) * in.ld + vcol + pp);
                    else
                        val_s[i] = 0.0f;
                }
            }
        } else {
            for (int i = tid; i < tb * NP; i += 128) {
                int tt = i / NP, nn = i - tt * NP;
                float kv = 0.0f, qv = 0.0f;
                if (nn < N) {
                    const float *row = src + (size_t)(c0 + tt) * in.ld + nn;
                    kv = add_partials(0.0f, row + kcol, in.S, in.stride);
                    if (in.silu)
                        kv = silu_f(kv);
                    if (MODE != 1) {
                        qv = add_partials(0.0f, row + qcol, in.S, in.stride);
                        if (in.silu)
                            qv = silu_f(qv);
                    }
                }
                key_s[i] = kv;
                if (MODE != 1)
                    qry_s[i] = qv;
            }
            for (int i = tid; i < tb * PT; i += 128) {
                int tt = i / PT, pp = i - tt * PT;
                float v = 0.0f;
                if (blockIdx.x * PT + pp < P) {
                    v = add_partials(0.0f, src + (size_t)(c0 + tt) * in.ld + vcol + pp, in.S, in.stride);
                    if (in.silu)
                        v = silu_f(v);
                }
                val_s[i] = v;
            }
        }
        if (tid < tb) {
            if (GATED) {
                if (in.coef_a != nullptr) {
                    a_s[tid] = in.coef_a[(size_t)(c0 + tid) * H + h];
                    b_s[tid] = in.coef_b[(size_t)(c0 + tid) * H + h];
                } else {
                    float i, f;
                    log_gates(in.gates, c0 + tid, h, i, f);
                    float mn = fmaxf(f + m_before, i);
                    a_s[tid] = expf(f + m_before - mn);
                    b_s[tid] = expf(i - mn);
                }
            } else if (in.dt != nullptr) {
                float d = add_partials(in.dt_bias[h], in.dt + (size_t)(c0 + tid) * in.dt_ld + in.dt_col0 + h, in.dt_S,
                                       in.dt_stride);
                d = softplus_f(d);
                a_s[tid] = expf(a_neg * d);
                b_s[tid] = d;
            } else {
                a_s[tid] = in.decay[h];
                b_s[tid] = 1.0f;
            }
        }
        if (direct)
            copy_async_wait();
        __syncthreads();
        if (MODE == 1) {
            // The piece's own end state needs no row's state in between: over the batch's rows
            // S <- (product of their decays) S + sum_s (b_s times the decays after s) k_s v_s^T,
            // the rows taken last to first so that the decays after a row are a running product.
            // One multiply-add a value and row instead of a multiply and a multiply-add.
            float all = 1.0f;
            for (int tt = 0; tt < tb; tt++)
                all *= a_s[tt];
            run *= all;
#pragma unroll
            for (int i = 0; i < NR; i++)
                s[i] *= all;
            float after = 1.0f;
            for (int tt = tb - 1; tt >= 0; tt--) {
                float wv = b_s[tt] * after * val_s[tt * PT + pl];
                after *= a_s[tt];
                const float4 *kk = reinterpret_cast<const float4 *>(key_s + tt * NP) + ns;
#pragma unroll
                for (int i4 = 0; i4 < NR / 4; i4++)
                    if (i4 < cnt4) {
                        float4 k4 = kk[i4 * nsplit];
                        s[4 * i4 + 0] = fmaf(wv, k4.x, s[4 * i4 + 0]);
                        s[4 * i4 + 1] = fmaf(wv, k4.y, s[4 * i4 + 1]);
                        s[4 * i4 + 2] = fmaf(wv, k4.z, s[4 * i4 + 2]);
                        s[4 * i4 + 3] = fmaf(wv, k4.w, s[4 * i4 + 3]);
                    }
            }
        } else
        for (int tt = 0; tt < tb; tt++) {
            float a = a_s[tt], v = val_s[tt * PT + pl], bv = b_s[tt] * v;
            const float4 *kk = reinterpret_cast<const float4 *>(key_s + tt * NP) + ns;
            const float4 *qq = reinterpret_cast<const float4 *>(qry_s + tt * NP) + ns;
            float4 ac = make_float4(0.0f, 0.0f, 0.0f, 0.0f);     // four chains, added at the end
            run *= a;
#pragma unroll
            for (int i4 = 0; i4 < NR / 4; i4++)
                if (i4 < cnt4) {
                    float4 k4 = kk[i4 * nsplit];
                    s[4 * i4 + 0] = fmaf(bv, k4.x, a * s[4 * i4 + 0]);
                    s[4 * i4 + 1] = fmaf(bv, k4.y, a * s[4 * i4 + 1]);
                    s[4 * i4 + 2] = fmaf(bv, k4.z, a * s[4 * i4 + 2]);
                    s[4 * i4 + 3] = fmaf(bv, k4.w, a * s[4 * i4 + 3]);
                    if (MODE != 1) {
                        float4 q4 = qq[i4 * nsplit];
                        ac.x = fmaf(s[4 * i4 + 0], q4.x, ac.x);
                        ac.y = fmaf(s[4 * i4 + 1], q4.y, ac.y);
                        ac.z = fmaf(s[4 * i4 + 2], q4.z, ac.z);
                        ac.w = fmaf(s[4 * i4 + 3], q4.w, ac.w);
                    }
                }
            if (MODE != 1) {
                float acc = (ac.x + ac.y) + (ac.z + ac.w);
                for (int o = 16; o >= PW; o >>= 1)
                    acc += __shfl_xor_sync(0xffffffffu, acc, o);
                if (ns == 0 && live)
                    y[(size_t)(c0 + tt) * H * P + (size_t)h * P + p] = GATED ? acc * in.q_scale : fmaf(dskip, v, acc);
            }
        }
    }
    // MODE 2: a sequence's last piece has walked the state to its end in the order of the one-pass
    // form; that is what the slot keeps (the carry pass's own end state differs from it in rounding)
    if (MODE == 2)
        st = slot + (size_t)h * per_head;
    if ((MODE != 2 || last_piece) && live) {
#pragma unroll
        for (int i = 0; i < NR; i++) {
            int nn = ((i >> 2) * nsplit + ns) * 4 + (i & 3);
            if (nn < N)
                st[(size_t)nn * P + p] = s[i];
        }
    }
    if (MODE == 1 && blockIdx.x == 0 && tid == 0)
        decays[(size_t)blockIdx.z * H + h] = run;
}

// Between the two passes over pieces: every sequence's state walks through its pieces,
// S <- decays[z] S + local[z], and local[z] is left holding the state its piece starts from
// (the state after the last piece is written by the second pass).  One thread per state value.
__global__ void __launch_bounds__(256)
matrix_state_carry_kernel(const float *state, size_t slot_stride, const int32_t *__restrict__ row_seq,
                          const int32_t *__restrict__ seq_slot, float *__restrict__ local,
                          const float *decays, int n, int H, size_t per_head, int piece, int pieces)
{
    pdl_trigger();
    int seq = blockIdx.y;
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)H * per_head)
        return;
    int h = (int)(idx / per_head);
    int rows = first_row_of(row_seq, n, seq + 1) - first_row_of(row_seq, n, seq);
    if (rows <= 0)
        return;
    int used = rows >= 2 * piece ? (rows + piece - 1) / piece : 1;
    const float *st = state + (size_t)seq_slot[seq] * slot_stride + idx;
    pdl_wait();
    float S = *st;
    // eight pieces' values are fetched together, then walked through in order
    for (int c0 = 0; c0 < used; c0 += 8) {
        float own[8], dec[8];
#pragma unroll
        for (int u = 0; u < 8; u++) {
            size_t z = (size_t)seq * pieces + min(c0 + u, used - 1);
            own[u] = local[z * H * per_head + idx];
            dec[u] = decays[z * H + h];
        }
#pragma unroll
        for (int u = 0; u < 8; u++)
            if (c0 + u < used) {
                size_t z = (size_t)seq * pieces + c0 + u;
                local[z * H * per_head + idx] = S;
                S = fmaf(dec[u], S, own[u]);
            }
    }
    (void)S;         // the slot's state is written by the second pass's last piece
}

// A gated memory's division ahead of the norm: part `part` of row r is first divided by
// max(|nq[r, part]|, e^(-m)) + floor.  em [n, parts] gives e^(-m); with em null (a decode step's rows) the
// gates are taken again from their sums and the running maximum in the slot's state, and the
// maximum after the row is written there.  nq null: no division.
struct PartScale {
    const float *nq, *em;
    float floor;
    LogGates gates;
    float *state;
    size_t slot_stride, m_off;
    const int32_t *row_seq, *seq_slot;
};

// where the running maximum of part `part` of row r stands that is to be written after every thread of
// the part has called part_factor (null: nowhere); reads the index arrays alone
__device__ __forceinline__ float *part_maximum(const PartScale &ps, int r, int part)
{
    if (ps.nq == nullptr || ps.em != nullptr)
        return nullptr;
    return ps.state + (size_t)ps.seq_slot[ps.row_seq[r]] * ps.slot_stride + ps.m_off + part;
}

// the factor on part `part` of row r; with mp the maximum after the row comes back in m
__device__ __forceinline__ float part_factor(const PartScale &ps, int r, int part, int parts, const float *mp, float &m)
{
    if (ps.nq == nullptr)
        return 1.0f;
    float e;
    if (ps.em != nullptr) {
        e = ps.em[(size_t)r * parts + part];
    } else {
        float i, f;
        log_gates(ps.gates, r, part, i, f);
        m = fmaxf(f + *mp, i);
        e = expf(-m);
    }
    return 1.0f / (fmaxf(fabsf(ps.nq[(size_t)r * parts + part]), e) + ps.floor);
}

// out[r, c] = rms_part(y[r, :] * pre)[c] * w[c] * post, where pre = silu of the sums in
// columns pre_col0.. of `pre` (null: 1), post = sigmoid (post_silu: silu) of the sums in columns
// post_col0.. of `post` (null: 1), w null is a weight of 1, and the row is normed in `parts` equal parts, each by its own root
// mean square.  A block per (row, part).
template <typename TO>
__global__ void __launch_bounds__(256)
gated_part_norm_kernel(const float *y, const float *pre, int pre_S, size_t pre_stride,
                       int pre_ld, int pre_col0, const float *post, int post_S, size_t post_stride,
                       int post_ld, int post_col0, const float *__restrict__ w, float eps, TO *__restrict__ out,
                       int width, int parts, int keep, int post_silu, PartScale ps)
{
    extern __shared__ float held[];          // the part's gated values, where they fit (keep != 0)
    __shared__ float red[32];
    pdl_trigger();
    int r = blockIdx.x, part = blockIdx.y, len = width / parts, c0 = part * len;
    float *mp = part_maximum(ps, r, part);
    pdl_wait();
    float ss = 0.0f, m_new = 0.0f;
    const float div = part_factor(ps, r, part, parts, mp, m_new);
    for (int c = c0 + threadIdx.x; c < c0 + len; c += blockDim.x) {
        float v = y[(size_t)r * width + c] * div;
        if (pre != nullptr)
            v *= silu_f(add_partials(0.0f, pre + (size_t)r * pre_ld + pre_col0 + c, pre_S, pre_stride));
        if (keep)
            held[c - c0] = v;
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    if (mp != nullptr && threadIdx.x == 0)
        *mp = m_new;           // every thread has read the old one: block_sum met them all
    float scale = 1.0f / sqrtf(ss / (float)len + eps);
    for (int c = c0 + threadIdx.x; c < c0 + len; c += blockDim.x) {
        float v;
        if (keep) {
            v = held[c - c0];
        } else {
            v = y[(size_t)r * width + c] * div;
            if (pre != nullptr)
                v *= silu_f(add_partials(0.0f, pre + (size_t)r * pre_ld + pre_col0 + c, pre_S, pre_stride));
        }
        v *= scale;
        if (w != nullptr)
            v *= w[c];
        if (post != nullptr) {
            float g = add_partials(0.0f, post + (size_t)r * post_ld + post_col0 + c, post_S, post_stride);
            v *= post_silu ? silu_f(g) : sigmoid_f(g);
        }
        out[(size_t)r * width + c] = from_f<TO>(v);
    }
}

// The same for short parts (a head's values each): a warp per (row, part), four neighbouring values
// a lane and up to U of those; lengths, columns and rows are multiples of four.
template <typename TO, int U>
__global__ void __launch_bounds__(256)
gated_part_norm_warp_kernel(const float *y, const float *pre, int pre_S, size_t pre_stride,
                            int pre_ld, int pre_col0, const float *post, int post_S, size_t post_stride,
                            int post_ld, int post_col0, const float *__restrict__ w, float eps, TO *__restrict__ out,
                            int width, int parts, int post_silu, unsigned tasks, PartScale ps)
{
    pdl_trigger();
    unsigned task = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (task >= tasks)
        return;
    int lane = threadIdx.x & 31;
    unsigned r = task / parts;
    int len = width / parts, c0 = (int)(task - r * parts) * len;
    auto sums4 = [](const float *p, int S, size_t stride) {
        float4 v = load4(p);
        for (int k = 1; k < S; k++) {
            float4 t = load4(p + (size_t)k * stride);
            v = make_float4(v.x + t.x, v.y + t.y, v.z + t.z, v.w + t.w);
        }
        return v;
    };
    float *mp = part_maximum(ps, (int)r, c0 / len);
    pdl_wait();
    float4 v[U], g[U];
    float ss = 0.0f, m_new = 0.0f;
    // y and the second gate are asked for before the factor is worked out
#pragma unroll
    for (int u = 0; u < U; u++) {
        int c = c0 + 4 * (lane + 32 * u);
        v[u] = g[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (c >= c0 + len)
            continue;
        v[u] = load4(y + (size_t)r * width + c);
        if (post != nullptr)
            g[u] = sums4(post + (size_t)r * post_ld + post_col0 + c, post_S, post_stride);
    }
    const float div = part_factor(ps, (int)r, c0 / len, parts, mp, m_new);
#pragma unroll
    for (int u = 0; u < U; u++) {
        int c = c0 + 4 * (lane + 32 * u);
        if (c >= c0 + len)
            continue;
        v[u] = make_float4(v[u].x * div, v[u].y * div, v[u].z * div, v[u].w * div);
        if (pre != nullptr) {
            float4 t = sums4(pre + (size_t)r * pre_ld + pre_col0 + c, pre_S, pre_stride);
            v[u] = make_float4(v[u].x * silu_f(t.x), v[u].y * silu_f(t.y), v[u].z * silu_f(t.z), v[u].w * silu_f(t.w));
        }
        ss = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, ss))));
    }
    ss = warp_sum(ss);
    if (mp != nullptr && lane == 0)
        *mp = m_new;           // every lane has read the old one: warp_sum met them all
    float scale = 1.0f / sqrtf(ss / (float)len + eps);
#pragma unroll
    for (int u = 0; u < U; u++) {
        int c = c0 + 4 * (lane + 32 * u);
        if (c >= c0 + len)
            continue;
        float4 o = make_float4(v[u].x * scale, v[u].y * scale, v[u].z * scale, v[u].w * scale);
        if (w != nullptr) {
            float4 t = load4(w + c);
            o = make_float4(o.x * t.x, o.y * t.y, o.z * t.z, o.w * t.w);
        }
        if (post != nullptr) {
            if (post_silu)
                o = make_float4(o.x * silu_f(g[u].x), o.y * silu_f(g[u].y), o.z * silu_f(g[u].z), o.w * silu_f(g[u].w));
            else
                o = make_float4(o.x * sigmoid_f(g[u].x), o.y * sigmoid_f(g[u].y), o.z * sigmoid_f(g[u].z),
                                o.w * sigmoid_f(g[u].w));
        }
        store4(out + (size_t)r * width + c, o);
    }
}

// q, k and v of a linear attention ahead of its recurrence, float32: out[r] = [q | k | v] from the
// sums' columns col0 .. (H D, H D and H Dv values), with the first 2 rot_half values of every q and
// k head turned (value i with value i + rot_half, angle tables [position, i]) and k times key_scale
// after that.  A thread has VEC neighbouring values, and where they turn their partners too.  VEC
// is 4 where D, Dv and rot_half are multiples of four and everything lies on 16-byte boundaries.
template <int VEC>
__device__ __forceinline__ void turn_load(const float *p, int S, size_t stride, float (&v)[VEC])
{
    if (VEC == 4) {
        float4 a = load4(p);
        for (int k = 1; k < S; k++) {
            float4 t = load4(p + (size_t)k * stride);
            a = make_float4(a.x + t.x, a.y + t.y, a.z + t.z, a.w + t.w);
        }
        v[0] = a.x; v[1 % VEC] = a.y; v[2 % VEC] = a.z; v[3 % VEC] = a.w;
    } else {
        v[0] = add_partials(0.0f, p, S, stride);
    }
}

template <int VEC>
__device__ __forceinline__ void turn_store(float *p, const float (&v)[VEC])
{
    if (VEC == 4)
        store4(p, make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]));
    else
        p[0] = v[0];
}

template <int VEC>
__global__ void __launch_bounds__(256)
turn_heads_kernel(const float *__restrict__ src, int S, size_t stride, int ld, int col0, int H, int D, int Dv,
                  const float *__restrict__ cs, const float *__restrict__ sn, int rot_half,
                  const int32_t *__restrict__ row_pos, float key_scale, float *__restrict__ out, int width,
                  int units)
{
    pdl_trigger();
    // a row's units: per q and k head the turned pairs, then the values that stay; then v
    int r = blockIdx.x, u = (int)(blockIdx.y * blockDim.x + threadIdx.x);
    if (u >= units)
        return;
    int pairs = rot_half / VEC, per = D / VEC - pairs;
    bool is_v = u >= 2 * H * per;
    int h = is_v ? 0 : u / per, i = is_v ? u - 2 * H * per : u - h * per;
    bool turned = !is_v && i < pairs;
    // the first value's column: pair i, or what lies behind the turned part
    int c = is_v ? 2 * H * D + i * VEC : h * D + (turned ? i : pairs + i) * VEC;
    float f = !is_v && h >= H ? key_scale : 1.0f;
    float co[VEC], si[VEC];
    if (turned) {
        size_t at = (size_t)row_pos[r] * rot_half + (size_t)i * VEC;
#pragma unroll
        for (int e = 0; e < VEC; e++) {
            co[e] = cs[at + e];
            si[e] = sn[at + e];
        }
    }
    pdl_wait();
    const float *p = src + (size_t)r * ld + col0 + c;
    float *dst = out + (size_t)r * width + c;
    float v[VEC], w[VEC];
    turn_load<VEC>(p, S, stride, v);
    if (turned) {
        turn_load<VEC>(p + rot_half, S, stride, w);
#pragma unroll
        for (int e = 0; e < VEC; e++) {
            float a = v[e], b = w[e];
            v[e] = fmaf(a, co[e], -(b * si[e]));
            w[e] = fmaf(b, co[e], a * si[e]) * f;
        }
        turn_store<VEC>(dst + rot_half, w);
    }
#pragma unroll
    for (int e = 0; e < VEC; e++)
        v[e] *= f;
    turn_store<VEC>(dst, v);
}

// The same for few rows: a cluster of C CTAs per (row, part), each with `cols` columns of the part
// held in shared memory; the CTAs exchange their sums of squares through one another's shared memory.
template <typename TO, int C>
__global__ void __launch_bounds__(256)
gated_part_norm_cluster_kernel(const float *y, const float *pre, int pre_S,
                               size_t pre_stride, int pre_ld, int pre_col0, const float *post,
                               int post_S, size_t post_stride, int post_ld, int post_col0,
                               const float *__restrict__ w, float eps, TO *__restrict__ out, int width, int parts,
                               int cols, int post_silu)
{
    extern __shared__ float held[];
    __shared__ float red[32];
    __shared__ float part_sq[C];
    pdl_trigger();
    uint32_t rank = cluster_rank();
    int idx = blockIdx.x / C, r = idx / parts, part = idx - r * parts, len = width / parts;
    int c0 = part * len + (int)rank * cols, c1 = min(part * len + len, c0 + cols);
    pdl_wait();
    float ss = 0.0f;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float v = y[(size_t)r * width + c];
        if (pre != nullptr)
            v *= silu_f(add_partials(0.0f, pre + (size_t)r * pre_ld + pre_col0 + c, pre_S, pre_stride));
        held[c - c0] = v;
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    if (threadIdx.x < C)
        cluster_write(&part_sq[rank], threadIdx.x, ss);
    cluster_arrive();
    cluster_wait();
    float tot = 0.0f;
#pragma unroll
    for (int k = 0; k < C; k++)
        tot += part_sq[k];
    float scale = 1.0f / sqrtf(tot / (float)len + eps);
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float v = held[c - c0] * scale;
        if (w != nullptr)
            v *= w[c];
        if (post != nullptr) {
            float g = add_partials(0.0f, post + (size_t)r * post_ld + post_col0 + c, post_S, post_stride);
            v *= post_silu ? silu_f(g) : sigmoid_f(g);
        }
        out[(size_t)r * width + c] = from_f<TO>(v);
    }
}

// Two mixers' results as one.  wl == null: out = sl * sum(L) + sr * sum(R).  Otherwise
// out = sl * rms(sum L) wl + sr * rms(sum R) wr (each normed over the whole row).
// A block per row; out: float32 [n, m].
__global__ void __launch_bounds__(256)
pair_combine_kernel(const float *L, int SL, size_t strideL, const float *R, int SR,
                    size_t strideR, const float *__restrict__ wl, const float *__restrict__ wr, float sl, float sr,
                    float eps, float *__restrict__ out, int m)
{
    __shared__ float red[32];
    pdl_trigger();
    int r = blockIdx.x;
    pdl_wait();
    float fl = sl, fr = sr;
    if (wl != nullptr) {
        float a = 0.0f, b = 0.0f;
        for (int c = threadIdx.x; c < m; c += blockDim.x) {
            float u = add_partials(0.0f, L + (size_t)r * m + c, SL, strideL);
            float v = add_partials(0.0f, R + (size_t)r * m + c, SR, strideR);
            a = fmaf(u, u, a);
            b = fmaf(v, v, b);
        }
        a = block_sum(a, red);
        b = block_sum(b, red);
        fl = 1.0f / sqrtf(a / (float)m + eps);
        fr = 1.0f / sqrtf(b / (float)m + eps);
    }
    for (int c = threadIdx.x; c < m; c += blockDim.x) {
        float u = add_partials(0.0f, L + (size_t)r * m + c, SL, strideL);
        float v = add_partials(0.0f, R + (size_t)r * m + c, SR, strideR);
        if (wl != nullptr)
            out[(size_t)r * m + c] = sl * ((u * fl) * wl[c]) + sr * ((v * fr) * wr[c]);
        else
            out[(size_t)r * m + c] = fmaf(fl, u, fr * v);
    }
}

// The same for few rows: a cluster of C CTAs per row, each with `cols` columns of it held in
// shared memory; the CTAs exchange their sums of squares through one another's shared memory.
template <int C>
__global__ void __launch_bounds__(256)
pair_combine_cluster_kernel(const float *L, int SL, size_t strideL, const float *R, int SR,
                            size_t strideR, const float *__restrict__ wl, const float *__restrict__ wr, float sl,
                            float sr, float eps, float *__restrict__ out, int m, int cols)
{
    extern __shared__ float both[];          // [2, cols]
    __shared__ float red[32];
    __shared__ float part_l[C], part_r[C];
    pdl_trigger();
    uint32_t rank = cluster_rank();
    int r = blockIdx.x / C;
    int c0 = (int)rank * cols, c1 = min(m, c0 + cols);
    pdl_wait();
    float a = 0.0f, b = 0.0f;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float u = add_partials(0.0f, L + (size_t)r * m + c, SL, strideL);
        float v = add_partials(0.0f, R + (size_t)r * m + c, SR, strideR);
        both[c - c0] = u;
        both[cols + c - c0] = v;
        a = fmaf(u, u, a);
        b = fmaf(v, v, b);
    }
    float fl = sl, fr = sr;
    if (wl != nullptr) {
        a = block_sum(a, red);
        b = block_sum(b, red);
        if (threadIdx.x < C) {
            cluster_write(&part_l[rank], threadIdx.x, a);
            cluster_write(&part_r[rank], threadIdx.x, b);
        }
        cluster_arrive();
        cluster_wait();
        float ta = 0.0f, tb = 0.0f;
#pragma unroll
        for (int k = 0; k < C; k++) {
            ta += part_l[k];
            tb += part_r[k];
        }
        fl = 1.0f / sqrtf(ta / (float)m + eps);
        fr = 1.0f / sqrtf(tb / (float)m + eps);
    } else {
        __syncthreads();
    }
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float u = both[c - c0], v = both[cols + c - c0];
        if (wl != nullptr)
            out[(size_t)r * m + c] = sl * ((u * fl) * wl[c]) + sr * ((v * fr) * wr[c]);
        else
            out[(size_t)r * m + c] = fmaf(fl, u, fr * v);
    }
}

// The weighted sum alone, four values a thread; everything on 16-byte boundaries.  The additions run
// in pair_combine_kernel's order.
__global__ void __launch_bounds__(256)
pair_sum_vec_kernel(const float *L, int SL, size_t strideL, const float *R, int SR, size_t strideR, float sl, float sr,
                    float *__restrict__ out, size_t fours)
{
    pdl_trigger();
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= fours)
        return;
    auto sums4 = [](const float *p, int S, size_t stride) {
        float4 v = load4(p);
        for (int k = 1; k < S; k++) {
            float4 t = load4(p + (size_t)k * stride);
            v = make_float4(v.x + t.x, v.y + t.y, v.z + t.z, v.w + t.w);
        }
        return v;
    };
    pdl_wait();
    float4 u = sums4(L + 4 * i, SL, strideL), v = sums4(R + 4 * i, SR, strideR);
    store4(out + 4 * i, make_float4(fmaf(sl, u.x, sr * v.x), fmaf(sl, u.y, sr * v.y), fmaf(sl, u.z, sr * v.z),
                                    fmaf(sl, u.w, sr * v.w)));
}

// g[r, j] = gelu_tanh(sum P[r, j]) * table[tokens[r], col0 + j]: a gate computed from the
// residual stream times the token's own vector for the layer.
template <typename TT, typename TO>
__global__ void __launch_bounds__(256)
token_gate_kernel(const float *__restrict__ P, int S, size_t stride, int ld, const TT *__restrict__ table,
                  int table_ld, int col0, const int32_t *__restrict__ tokens, TO *__restrict__ out, int n, int dim)
{
    pdl_trigger();
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)n * dim)
        return;
    int r = (int)(idx / dim), j = (int)(idx - (size_t)r * dim);
    float e = to_f(table[(size_t)tokens[r] * table_ld + col0 + j]);
    pdl_wait();
    float v = add_partials(0.0f, P + (size_t)r * ld + j, S, stride);
    float u = 0.7978845608028654f * fmaf(0.044715f * v * v, v, v);
    out[idx] = from_f<TO>(0.5f * v * (1.0f + tanhf(u)) * e);
}

}  // namespace jb

using namespace jb;

// Into how many lanes a column of the state is split: the fewest that leave at most per_lane
// state values to a lane, more while a block's 128 / nsplit columns are more than twice P.
static int scan_nsplit(int N, int P, int per_lane)
{
    int ns = 1;
    while (ns < 32 && ((N + 4 * ns - 1) / (4 * ns)) * 4 > per_lane)
        ns *= 2;
    while (ns < 32 && 128 / ns >= 2 * P)
        ns *= 2;
    return ns;
}

// rows to a piece when long sequences are cut into pieces that run side by side
extern "C" int jb_matrix_state_piece(void) { return 128; }
// Floats of scratch for a step whose longest sequence brings max_len rows (0: one pass does it).
static long long matrix_scratch(int n_seqs, int max_len, int H, size_t per_head)
{
    int piece = jb_matrix_state_piece();
    if (max_len < 2 * piece)
        return 0;
    long long pieces = (max_len + piece - 1) / piece;
    long long need = (long long)n_seqs * pieces * ((long long)H * (long long)per_head + H);
    return need > (1ll << 28) ? 0 : need;       // more than 1 GiB of scratch: one pass after all
}
extern "C" long long jb_matrix_state_scratch(int n_seqs, int max_len, int H, int N, int P)
{
    return matrix_scratch(n_seqs, max_len, H, (size_t)N * P);
}

static int scan_launch(const ScanIn &in, bool gated, float *state, long long slot_stride, const int32_t *row_seq,
                       const int32_t *seq_slot, float *y, int n, int n_seqs, int H, int G, int N, int P,
                       int every_row_starts, float *scratch, int max_len, cudaStream_t st)
{
    // 16 state values to a lane (more blocks, fewer registers, a shorter chain per row) where 32
    // lanes to a column are enough for that; 32 otherwise
    // (a decode step's one row per sequence moves the state and little else: fewer lanes to a
    // column then, so that a warp reads 32 bytes of a state row at a time)
    bool small = N <= 16 * 32 && !every_row_starts;
    int nsplit = scan_nsplit(N, P, small ? 16 : 32);
    if (((N + 4 * nsplit - 1) / (4 * nsplit)) * 4 > 32)
        return JB_EINVAL;
    constexpr int TB = 16;
    int PT = 128 / nsplit;
    int NP = (N + 4 * nsplit - 1) / (4 * nsplit) * (4 * nsplit);
    unsigned ptiles = (unsigned)((P + PT - 1) / PT) + (gated ? 1u : 0u);     // gated: a block more for n
    size_t smem = (size_t)TB * (2 * NP + PT + 2) * 4;
    const size_t per_head = (size_t)N * P + (gated ? N : 0);
    int piece = jb_matrix_state_piece();
    bool whole = scratch == nullptr || every_row_starts || matrix_scratch(n_seqs, max_len, H, per_head) == 0;
    int pieces = whole ? 1 : (max_len + piece - 1) / piece;
    if ((long long)n_seqs * pieces > 65535)
        return JB_EINVAL;
    float *local = scratch, *decays = whole ? nullptr : scratch + (size_t)n_seqs * pieces * H * per_head;
    dim3 grid(ptiles, (unsigned)H, (unsigned)(n_seqs * pieces));
#define JB_SCAN_G(NRV, MODE, NSV, GT, SMEM)                                                                        \
    do {                                                                                                       \
        if ((SMEM) > 48 * 1024) {                                                                              \
            /* long states: the rows in shared memory need more than a kernel gets unasked */                  \
            static const bool asked = cudaFuncSetAttribute(matrix_state_scan_kernel<NRV, TB, MODE, NSV, GT>,   \
                                                           cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                                                           160 * 1024) == cudaSuccess;                         \
            (void)asked;                                                                                       \
        }                                                                                                      \
        launch(matrix_state_scan_kernel<NRV, TB, MODE, NSV, GT>, grid, 128, (SMEM), st, in, state,                 \
               (size_t)slot_stride, row_seq, seq_slot, y, local, decays, n, H, G, N, P, nsplit,                \
               whole ? every_row_starts : 0, whole ? 0 : piece, pieces);                                       \
    } while (0)
#define JB_SCAN_N(NRV, MODE, NSV, SMEM)                                        \
    do {                                                                       \
        if (gated) JB_SCAN_G(NRV, MODE, NSV, true, SMEM);                      \
        else JB_SCAN_G(NRV, MODE, NSV, false, SMEM);                           \
    } while (0)
    // the commonest shapes have kernels of their own: 128 or 64 state rows, 16 to a lane (prompts),
    // 128 rows, 32 to a lane (decode rows)
#define JB_SCAN(MODE, SMEM)                                              \
    do {                                                                 \
        if (small && nsplit == 8 && N == 128) JB_SCAN_N(16, MODE, 8, SMEM); \
        else if (small && nsplit == 4 && N == 64) JB_SCAN_N(16, MODE, 4, SMEM); \
        else if (!small && nsplit == 4 && N == 128) JB_SCAN_N(32, MODE, 4, SMEM); \
        else if (small) JB_SCAN_N(16, MODE, 0, SMEM);                    \
        else JB_SCAN_N(32, MODE, 0, SMEM);                               \
    } while (0)
    if (whole) {
        JB_SCAN(0, smem);
        return launch_status();
    }
    size_t smem1 = (size_t)TB * (NP + PT + 2) * 4;
    JB_SCAN(1, smem1);
    launch(matrix_state_carry_kernel, dim3((unsigned)(((size_t)H * per_head + 255) / 256), (unsigned)n_seqs), 256, 0, st,
           (const float *)state, (size_t)slot_stride, row_seq, seq_slot, local, (const float *)decays, n, H, per_head, piece, pieces);
    JB_SCAN(2, smem);
#undef JB_SCAN
#undef JB_SCAN_N
#undef JB_SCAN_G
    return launch_status();
}

// src: float32 [S, n, ld] holding v (H P columns from val_col0), k and q (G N columns each);
// with dt (sums [dt_S, n, dt_ld], H columns from dt_col0) the selective form, otherwise
// decay [H].  state: [H, N, P] per slot.  y: float32 [n, H P].  scratch (with max_len, the most
// rows a sequence brings): jb_matrix_state_scratch floats, or null for one pass.
extern "C" int jb_matrix_state_scan(const float *src, int S, long long stride, int ld, int val_col0, int key_col0,
                                    int qry_col0, int silu, const float *dt, int dt_S, long long dt_stride,
                                    int dt_ld, int dt_col0, const float *dt_bias, const float *a_log,
                                    const float *skip, const float *decay, float *state, long long slot_stride,
                                    const int32_t *row_seq, const int32_t *seq_slot, float *y, int n, int n_seqs,
                                    int H, int G, int N, int P, int every_row_starts, float *scratch, int max_len,
                                    cudaStream_t st)
{
    if (n <= 0 || n_seqs <= 0)
        return JB_OK;
    if (H <= 0 || G <= 0 || H % G || N <= 0 || N > 1024 || P <= 0 || S <= 0 || src == nullptr || state == nullptr ||
        y == nullptr || (dt != nullptr && (dt_bias == nullptr || a_log == nullptr || dt_S <= 0)) ||
        (dt == nullptr && decay == nullptr) || H > 65535 || n_seqs > 65535 ||
        ld < val_col0 + H * P || ld < key_col0 + G * N || ld < qry_col0 + G * N)
        return JB_EINVAL;
    ScanIn in{src, S, (size_t)stride, ld, val_col0, key_col0, qry_col0, silu, dt, dt_S, (size_t)dt_stride, dt_ld,
              dt_col0, dt_bias, a_log, skip, decay, nullptr, nullptr, LogGates(), 1.0f, nullptr};
    return scan_launch(in, false, state, slot_stride, row_seq, seq_slot, y, n, n_seqs, H, G, N, P, every_row_starts,
                       scratch, max_len, st);
}

// Floats of scratch of jb_gated_memory_scan: the gates' a and b per row and head (not in a decode
// step), then what the pieces need.
extern "C" long long jb_gated_memory_scratch(int n, int n_seqs, int max_len, int H, int N, int P, int every_row_starts)
{
    if (every_row_starts)
        return 0;
    return 2ll * n * H + matrix_scratch(n_seqs, max_len, H, (size_t)N * P + N);
}

// The gated memory's recurrence.  src: float32 [S, n, ld] holding v (H P columns), k and q (H N each) and
// the two log gates (H each); i_bias, f_bias [H].  state per slot: [H, (N P | N)] and [H] running maxima.
// y: [n, H P] and nq: [n, H], both times q_scale and not yet divided.  em: [n, H], e^(-m), written
// unless every row starts (a decode step: the norm that follows takes the gates again and
// writes the running maxima).
extern "C" int jb_gated_memory_scan(const float *src, int S, long long stride, int ld, int val_col0, int key_col0,
                                    int qry_col0, int i_col0, int f_col0, const float *i_bias, const float *f_bias,
                                    float cap, float q_scale, float *state, long long slot_stride,
                                    const int32_t *row_seq, const int32_t *seq_slot, float *y, float *nq, float *em,
                                    int n, int n_seqs, int H, int N, int P, int every_row_starts, float *scratch,
                                    int max_len, cudaStream_t st)
{
    if (n <= 0 || n_seqs <= 0)
        return JB_OK;
    if (H <= 0 || N <= 0 || N > 1024 || P <= 0 || S <= 0 || src == nullptr || state == nullptr || y == nullptr ||
        nq == nullptr || i_bias == nullptr || f_bias == nullptr || !(cap > 0.0f) || H > 65535 || n_seqs > 65535 ||
        (!every_row_starts && (scratch == nullptr || em == nullptr)) || ld < val_col0 + H * P || ld < key_col0 + H * N ||
        ld < qry_col0 + H * N || ld < i_col0 + H || ld < f_col0 + H)
        return JB_EINVAL;
    LogGates g{src, S, (size_t)stride, ld, i_col0, f_col0, i_bias, f_bias, cap};
    ScanIn in{src, S, (size_t)stride, ld, val_col0, key_col0, qry_col0, 0, nullptr, 0, 0, 0,
              0, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, g, q_scale, nq};
    if (!every_row_starts) {
        size_t m_off = (size_t)H * ((size_t)N * P + N);
        float *ca = scratch, *cb = scratch + (size_t)n * H;
        // (LG_THREADS threads take a sequence's rows; the host may not know how long the longest is)
        dim3 gg((unsigned)H, (unsigned)n_seqs);
        int per = ((max_len > 0 ? max_len : n) + LG_THREADS - 1) / LG_THREADS;
#define JB_LG(HELD)                                                                                             \
    launch(log_gates_kernel<HELD>, gg, LG_THREADS, 0, st, g, state, (size_t)slot_stride, m_off, row_seq, seq_slot, ca, cb, em, n, H)
        if (per <= 1) JB_LG(1);
        else if (per <= 4) JB_LG(4);
        else if (per <= 8) JB_LG(8);
        else JB_LG(0);
#undef JB_LG
        in.coef_a = ca;
        in.coef_b = cb;
        scratch += 2 * (size_t)n * H;
        if (matrix_scratch(n_seqs, max_len, H, (size_t)N * P + N) == 0)
            scratch = nullptr;
    }
    return scan_launch(in, true, state, slot_stride, row_seq, seq_slot, y, n, n_seqs, H, H, N, P, every_row_starts,
                       scratch, max_len, st);
}

static int part_norm_launch(const float *y, const float *pre, int pre_S, long long pre_stride, int pre_ld,
                                  int pre_col0, const float *post, int post_S, long long post_stride, int post_ld,
                                  int post_col0, int post_silu, const float *w, float eps, void *out, int out_dt,
                                  int n, int width, int parts, int few_rows, const PartScale &ps, cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (width <= 0 || parts <= 0 || width % parts || parts > 65535 || y == nullptr ||
        (pre != nullptr && (pre_S <= 0 || pre_ld < pre_col0 + width)) ||
        (post != nullptr && (post_S <= 0 || post_ld < post_col0 + width)))
        return JB_EINVAL;
    if (few_rows && ps.nq == nullptr && n * parts <= 64 && width / parts >= 512 && out_dt == JB_BF16) {
        // few blocks otherwise: a cluster of CTAs per (row, part)
        constexpr int C = 4;
        int cols = (width / parts + C - 1) / C;
        if ((size_t)cols * 4 <= 40 * 1024) {
            launch_cluster(gated_part_norm_cluster_kernel<bf16, C>, dim3((unsigned)(n * parts * C)), 256, (size_t)cols * 4,
                           st, C, y, pre, pre_S, (size_t)pre_stride, pre_ld, pre_col0, post, post_S, (size_t)post_stride,
                           post_ld, post_col0, w, eps, (bf16 *)out, width, parts, cols, post_silu);
            return launch_status();
        }
    }
    dim3 grid((unsigned)n, (unsigned)parts);
    size_t len = (size_t)(width / parts);
    // short parts of which a row has several: a warp each
    auto four = [](const float *p, int ld, long long stride, int col0) {
        return p == nullptr || ((uintptr_t)p % 16 == 0 && ld % 4 == 0 && stride % 4 == 0 && col0 % 4 == 0);
    };
    if (parts > 1 && len % 4 == 0 && len <= 256 && (long long)n * parts <= 0x7fffffffll && four(y, width, 0, 0) &&
        four(w, 4, 0, 0) && four(pre, pre_ld, pre_stride, pre_col0) && four(post, post_ld, post_stride, post_col0) &&
        (uintptr_t)out % 16 == 0 && (out_dt == JB_F32 || out_dt == JB_BF16)) {
        unsigned tasks = (unsigned)n * (unsigned)parts;
        const int warps = n <= 64 ? 2 : 8;          // few rows: more blocks
        unsigned g = (tasks + warps - 1) / warps;
#define JB_GPN(TO, U)                                                                                          \
    launch(gated_part_norm_warp_kernel<TO, U>, g, 32 * warps, 0, st, y, pre, pre_S, (size_t)pre_stride, pre_ld,  \
           pre_col0, post, post_S, (size_t)post_stride, post_ld, post_col0, w, eps, (TO *)out, width, parts,     \
           post_silu, tasks, ps)
        if (out_dt == JB_F32) {
            if (len <= 128) JB_GPN(float, 1); else JB_GPN(float, 2);
        } else {
            if (len <= 128) JB_GPN(bf16, 1); else JB_GPN(bf16, 2);
        }
#undef JB_GPN
        return launch_status();
    }
    int keep = len * 4 <= 40 * 1024 ? 1 : 0;
    size_t smem = keep ? len * 4 : 0;
    int threads = len >= 1024 ? 256 : 128;
    if (out_dt == JB_F32)
        launch(gated_part_norm_kernel<float>, grid, threads, smem, st, y, pre, pre_S, (size_t)pre_stride, pre_ld, pre_col0,
               post, post_S, (size_t)post_stride, post_ld, post_col0, w, eps, (float *)out, width, parts, keep, post_silu, ps);
    else if (out_dt == JB_BF16)
        launch(gated_part_norm_kernel<bf16>, grid, threads, smem, st, y, pre, pre_S, (size_t)pre_stride, pre_ld, pre_col0,
               post, post_S, (size_t)post_stride, post_ld, post_col0, w, eps, (bf16 *)out, width, parts, keep, post_silu, ps);
    else
        return JB_EINVAL;
    return launch_status();
}

extern "C" int jb_gated_part_norm(const float *y, const float *pre, int pre_S, long long pre_stride, int pre_ld,
                                  int pre_col0, const float *post, int post_S, long long post_stride, int post_ld,
                                  int post_col0, int post_silu, const float *w, float eps, void *out, int out_dt,
                                  int n, int width, int parts, int few_rows, cudaStream_t st)
{
    return part_norm_launch(y, pre, pre_S, pre_stride, pre_ld, pre_col0, post, post_S, post_stride, post_ld, post_col0,
                            post_silu, w, eps, out, out_dt, n, width, parts, few_rows, PartScale(), st);
}

// What follows jb_gated_memory_scan: y [n, H P] divided per head by max(|nq|, e^(-m)) + floor, each head
// RMS-normed, times w [H P], times the sigmoid of the sums in columns g_col0.. of src.  em as the scan
// left it, or null for a decode step's rows (then the gates' sums and the state, as the scan took them).
extern "C" int jb_gated_memory_norm(const float *y, const float *nq, const float *em, float floor, const float *src,
                                    int S, long long stride, int ld, int g_col0, int i_col0, int f_col0,
                                    const float *i_bias, const float *f_bias, float cap, float *state,
                                    long long slot_stride, const int32_t *row_seq, const int32_t *seq_slot,
                                    const float *w, float eps, void *out, int out_dt, int n, int H, int N, int P,
                                    cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (nq == nullptr || src == nullptr || S <= 0 || H <= 0 || N <= 0 || P <= 0 || ld < g_col0 + H * P ||
        (em == nullptr && (state == nullptr || i_bias == nullptr || f_bias == nullptr || row_seq == nullptr ||
                           seq_slot == nullptr || ld < i_col0 + H || ld < f_col0 + H || !(cap > 0.0f))))
        return JB_EINVAL;
    PartScale ps{nq, em, floor, LogGates{src, S, (size_t)stride, ld, i_col0, f_col0, i_bias, f_bias, cap}, state,
                 (size_t)slot_stride, (size_t)H * ((size_t)N * P + N), row_seq, seq_slot};
    return part_norm_launch(y, nullptr, 0, 0, 0, 0, src, S, stride, ld, g_col0, 0, w, eps, out, out_dt, n, H * P, H, 0,
                            ps, st);
}

// src: sums [S, n, ld]; out: float32 [n, 2 H D + H Dv].  See turn_heads_kernel.
extern "C" int jb_turn_heads(const float *src, int S, long long stride, int ld, int col0, int H, int D, int Dv,
                             const float *cs, const float *sn, int rot_half, const int32_t *row_pos, float key_scale,
                             float *out, int n, cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    long long width = (long long)H * (2 * D + Dv);
    if (src == nullptr || out == nullptr || S <= 0 || H <= 0 || D <= 0 || Dv <= 0 || rot_half < 0 || 2 * rot_half > D ||
        col0 < 0 || col0 + width > ld || (rot_half > 0 && (cs == nullptr || sn == nullptr || row_pos == nullptr)))
        return JB_EINVAL;
    bool vec = D % 4 == 0 && Dv % 4 == 0 && rot_half % 4 == 0 && ld % 4 == 0 && stride % 4 == 0 && col0 % 4 == 0 &&
               (uintptr_t)src % 16 == 0 && (uintptr_t)out % 16 == 0;
    const int V = vec ? 4 : 1;
    long long units = 2ll * H * (D / V - rot_half / V) + (long long)H * (Dv / V);
    // few rows: smaller blocks, so that a row's units spread over more SMs
    const int threads = n <= 64 ? 64 : 256;
    if ((units + threads - 1) / threads > 65535)
        return JB_EINVAL;
    dim3 grid((unsigned)n, (unsigned)((units + threads - 1) / threads));
    if (vec)
        launch(turn_heads_kernel<4>, grid, threads, 0, st, src, S, (size_t)stride, ld, col0, H, D, Dv, cs, sn, rot_half,
               row_pos, key_scale, out, (int)width, (int)units);
    else
        launch(turn_heads_kernel<1>, grid, threads, 0, st, src, S, (size_t)stride, ld, col0, H, D, Dv, cs, sn, rot_half,
               row_pos, key_scale, out, (int)width, (int)units);
    return launch_status();
}

extern "C" int jb_pair_combine(const float *L, int SL, long long strideL, const float *R, int SR, long long strideR,
                               const float *wl, const float *wr, float sl, float sr, float eps, float *out, int n,
                               int m, int few_rows, cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (m <= 0 || SL <= 0 || SR <= 0 || L == nullptr || R == nullptr || out == nullptr || (wl == nullptr) != (wr == nullptr))
        return JB_EINVAL;
    // (a decode step's products leave many partial sums a value: the cluster kernel's threads share them out)
    if (wl == nullptr && !(few_rows && n <= 32 && m >= 512) && m % 4 == 0 && strideL % 4 == 0 && strideR % 4 == 0 &&
        (((uintptr_t)L | (uintptr_t)R | (uintptr_t)out) & 15) == 0) {
        size_t fours = (size_t)n * m / 4;
        unsigned threads = fours < 148 * 256 ? 64 : 256;       // few rows: more blocks
        launch(pair_sum_vec_kernel, (unsigned)((fours + threads - 1) / threads), threads, 0, st, L, SL, (size_t)strideL, R, SR,
               (size_t)strideR, sl, sr, out, fours);
        return launch_status();
    }
    if (few_rows && n <= 32 && m >= 512) {
        constexpr int C = 8;
        int cols = (m + C - 1) / C;
        if ((size_t)cols * 8 <= 40 * 1024) {
            launch_cluster(pair_combine_cluster_kernel<C>, dim3((unsigned)n * C), 256, (size_t)cols * 8, st, C, L, SL,
                           (size_t)strideL, R, SR, (size_t)strideR, wl, wr, sl, sr, eps, out, m, cols);
            return launch_status();
        }
    }
    launch(pair_combine_kernel, (unsigned)n, 256, 0, st, L, SL, (size_t)strideL, R, SR, (size_t)strideR, wl, wr, sl, sr,
           eps, out, m);
    return launch_status();
}

extern "C" int jb_token_gate(const float *P, int S, long long stride, int ld, const void *table, int table_dt,
                             int table_ld, int col0, const int32_t *tokens, void *out, int out_dt, int n, int dim,
                             cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (dim <= 0 || ld < dim || table_ld < col0 + dim || col0 < 0 || S <= 0 || P == nullptr || table == nullptr ||
        tokens == nullptr)
        return JB_EINVAL;
    unsigned grid = (unsigned)(((size_t)n * dim + 255) / 256);
#define JB_TG(TT, TO)                                                                                          \
    launch(token_gate_kernel<TT, TO>, grid, 256, 0, st, P, S, (size_t)stride, ld, (const TT *)table, table_ld, \
           col0, tokens, (TO *)out, n, dim)
    if (table_dt == JB_F32 && out_dt == JB_F32) JB_TG(float, float);
    else if (table_dt == JB_BF16 && out_dt == JB_BF16) JB_TG(bf16, bf16);
    else if (table_dt == JB_F32 && out_dt == JB_BF16) JB_TG(float, bf16);
    else if (table_dt == JB_BF16 && out_dt == JB_F32) JB_TG(bf16, float);
    else return JB_EINVAL;
#undef JB_TG
    return launch_status();
}
