// A state-space recurrence with one decay per head and token (Mamba-2), for mixed batches of prompt portions and
// single tokens, with the state of every request in slots of two state tensors.
//
// A row of projections holds [z: H dv | x: H dv | B: G N | C: G N | dt: H].  x, B and C together pass a causal convolution
// per channel and silu; then, per head h with its group g = h / (H / G) and a state S [N][dv] that starts at zero,
//
//     dt  = softplus(dt + dt_bias)            a_t = exp(-exp(A_log) dt_t)
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T      y_t = (S_t^T C_t + D x_t) * silu(z_t)
//
// and y is RMS-normed in equal parts of the row, times a gain.  Everything is float32; the normed row alone is stored in the
// model's type.  (In bfloat16 models portions round x, B and C to it behind silu, where their sizes suit the tensor cores.)
//
// The convolution's inputs of the last `taps` positions live in a ring [taps][channels] per request, position p in entry
// p mod taps: a step writes the entry of its own position and reads the others, so CTAs that share channels do not
// depend on one another.
//
// Steps in which every request brings one row take one kernel (step_kernel) and the norm: a CTA per (slice of value
// channels, head, request) forms its own channels of the convolution, updates its part of the state in registers
// (requested before the projections are waited for) and gates its values.
//
// Steps with portions cut a request's rows into chunks of kC rows.  With c_i the sum of the chunk's decay logarithms
// up to and including row i,
//
//     y_i   = exp(c_i) C_i^T S_in + sum over j <= i of (C_i . B_j) exp(c_i - c_j) dt_j x_j
//     S_out = exp(c_last) S_in + sum over j of exp(c_last - c_j) dt_j B_j x_j^T
//
//   conv_kernel    convolution and silu of every channel; dt and the c_i of every head
//   ring_kernel    the ring takes the portions' last inputs
//   pairs_kernel   C_i . B_j per (chunk, group), which the group's heads share
//   outer_kernel   every chunk's own addition to the state
//   carry_kernel   the states at the chunks' starts, element by element over a request's chunks in order;
//                  moves the slot on
//   apply_kernel   y of every chunk, with D and the gate
//   part_norm_kernel
// In bfloat16 models with N and dv in steps of 16 the products run on the tensor cores (mma.sync m16n8k16, chunks of kT
// rows): x, B and C are bfloat16, and what is float32 enters as two bfloat16 terms, high and low (16 bits of mantissa):
//
//   outer_tc_kernel   B^T (exp(c_last - c_j) dt_j x_j), the weighted rows split
//   carry_kernel      leaves the states at the chunks' starts split, float32 in the slot and in every sum
//   apply_tc_kernel   C S_in with the state split, rows times exp(c_i); then, key tile by key tile, C B^T in registers, times the
//                     float32 decays and steps, split, times x
// The c_i may reach tens of thousands while their differences are small: they are summed in double precision and
// kept as two floats, whose differences are formed pairwise.  Where a prompt is cut changes the order of float32 sums and
// nothing else.
#include "common.cuh"

KLLM_EXPORT_LAST_ERROR(ssd)

namespace {

constexpr int kC = 64;          // rows of a chunk
constexpr int kT = 128;         // ... of the tensor-core form
constexpr int kThreads = 256;

struct SsdArgs {
    const float* proj;                      // [n] rows at `stride`
    int64_t stride;
    const float *conv_w, *conv_b;           // [channels][taps], [channels]
    const float *dt_bias, *a_log, *d;       // [H]
    int taps, heads, groups, N, dv, inner, channels;
    const int *q_start, *start_pos, *state_slots;
    int n_requests;
    float* state;                           // [slots][state_stride]: S as [H][N][dv]
    int64_t state_stride;
    float* ring;                            // [slots][ring_stride]: [taps][ch_pad]
    int64_t ring_stride;
    int ch_pad;                             // channels rounded up to a multiple of 4: row length of ring and xc
    float* y;                               // [n][inner]: gated, before the norm
    // work of the form for portions
    void* xc;                               // [n][xc_pad] float32, or bfloat16 in the tensor-core form: x, B, C behind the convolution
    int xc_pad;
    float* dt;                              // [chunks][H][rows of a chunk]
    float2* cum;                            // [chunks][H][rows of a chunk]
    float* pairs;                           // [chunks][G][kC][kC]
    float* s_in;                            // [chunks][H][N][dv]
    bf16* s_split;                          // tensor-core form: [2][chunks][H][N][dv], high and low terms
    int64_t split_plane;                    // elements of one of the two
    bool vec;                               // sizes and addresses allow 16-byte accesses
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// exp(a - b) of two sums kept as (high, low)
__device__ __forceinline__ float exp_diff(float2 a, float2 b) { return expf((a.x - b.x) + (a.y - b.y)); }

template <int V> struct Vec { float x[V]; };
template <int V> __device__ __forceinline__ Vec<V> load_vec(const float* p) {
    Vec<V> r;
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.x[0] = t.x; r.x[1] = t.y; r.x[2] = t.z; r.x[3] = t.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; i++) r.x[i] = p[i];
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_vec(float* p, const Vec<V>& r) {
    if constexpr (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r.x[0], r.x[1], r.x[2], r.x[3]);
    } else {
#pragma unroll
        for (int i = 0; i < V; i++) p[i] = r.x[i];
    }
}

// ---- one row per request -----------------------------------------------------------------------------------
// grid (slices, heads, requests).  Thread (cg, nl): V value channels e0 + cg V ..., state channels nl, nl + lanes, ...
// Shared memory: partial sums [kThreads * V], x [sl], B [N], C [N].  Started early, the kernel reads state and ring before
// the kernel in front of it has ended: that kernel must write neither.
template <int V>
__global__ void __launch_bounds__(kThreads, 4)
step_kernel(const SsdArgs a, int sl) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NB = V == 4 ? 8 : 16;                     // state channels in flight per thread
    const int tid = threadIdx.x, slice = blockIdx.x, head = blockIdx.y, req = blockIdx.z;
    const int N = a.N, dv = a.dv, per = a.heads / a.groups, group = head / per;
    float* ps = sm;                                         // [kThreads * V], 16-byte aligned
    float* xs = ps + kThreads * V;                          // [sl], a multiple of V
    float* bs = xs + sl;                                    // B [N], then C [N]
    const int t = a.q_start[req], p = a.start_pos[req], slot = a.state_slots[req];
    const int nv = sl / V, lanes = kThreads / nv, cg = tid % nv, nl = tid / nv;
    const bool on = nl < lanes;
    const int e = slice * sl + cg * V;
    float* Sg = a.state + (int64_t)slot * a.state_stride + (int64_t)head * N * dv + e;
    Vec<V> s[NB];
#pragma unroll
    for (int i = 0; i < NB; i++) {
        const int n = nl + i * lanes;
        if (on && n < N) s[i] = load_vec<V>(Sg + (int64_t)n * dv);
    }
    float* ring = a.ring + (int64_t)slot * a.ring_stride;
    const int mine = sl + 2 * N;                            // channels that this CTA convolves: x slice, B, C
    auto channel = [&](int i) {
        return i < sl ? head * dv + slice * sl + i : i < sl + N ? a.inner + group * N + (i - sl)
                                                               : a.inner + a.groups * N + group * N + (i - sl - N);
    };
    // what earlier rows put into a channel's sum: of the first kEarly channels of a thread before the projections are waited
    // for, all loads of four taps at once
    auto before = [&](int c) {
        float v = a.conv_b[c];
        const float* w = a.conv_w + (int64_t)c * a.taps;
        for (int i0 = 0; i0 < a.taps - 1; i0 += 4) {
            float wv[4], rv[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const int i = i0 + u, q = p - (a.taps - 1) + i;
                const bool in = i < a.taps - 1 && q >= 0;
                wv[u] = in ? w[i] : 0.f;
                rv[u] = in ? ring[(int64_t)(q % a.taps) * a.ch_pad + c] : 0.f;
            }
#pragma unroll
            for (int u = 0; u < 4; u++) v = fmaf(wv[u], rv[u], v);
        }
        return v;
    };
    constexpr int kEarly = 2;
    float sum[kEarly], wlast[kEarly];
    int ch[kEarly];
#pragma unroll
    for (int u = 0; u < kEarly; u++) {
        const int i = tid + u * kThreads;
        ch[u] = i < mine ? channel(i) : -1;
        sum[u] = ch[u] >= 0 ? before(ch[u]) : 0.f;
        wlast[u] = ch[u] >= 0 ? a.conv_w[(int64_t)ch[u] * a.taps + a.taps - 1] : 0.f;
    }
    const float rate = expf(a.a_log[head]), dbias = a.dt_bias[head], dskip = a.d[head];
    griddep_wait();
    griddep_launch();
    const float* row = a.proj + (int64_t)t * a.stride;
    const float* u_row = row + a.inner;
    float in[kEarly];
#pragma unroll
    for (int u = 0; u < kEarly; u++) in[u] = ch[u] >= 0 ? u_row[ch[u]] : 0.f;
    const float dt_in = row[a.inner + a.channels + head];
    const float* z = row + head * dv + slice * sl;
    const float z_first = tid < sl ? z[tid] : 0.f;
    auto keep = [&](int i, int c, float x, float v) {
        xs[i] = silu_f(v);                                  // x slice, B and C lie one behind the other
        // one CTA moves each channel's ring on: x its own, B and C the group's first head
        if (i < sl || (slice == 0 && head == group * per)) ring[(int64_t)(p % a.taps) * a.ch_pad + c] = x;
    };
#pragma unroll
    for (int u = 0; u < kEarly; u++)
        if (ch[u] >= 0) keep(tid + u * kThreads, ch[u], in[u], fmaf(wlast[u], in[u], sum[u]));
    for (int i = tid + kEarly * kThreads; i < mine; i += kThreads) {
        const int c = channel(i);
        const float x = u_row[c];
        keep(i, c, x, fmaf(a.conv_w[(int64_t)c * a.taps + a.taps - 1], x, before(c)));
    }
    const float dt = softplus_f(dt_in + dbias);
    const float al = expf(-rate * dt);
    __syncthreads();
    if (on) {
        Vec<V> xv, acc;
#pragma unroll
        for (int j = 0; j < V; j++) {
            xv.x[j] = xs[cg * V + j] * dt;
            acc.x[j] = 0.f;
        }
        const float* cs = bs + N;
        for (int n0 = nl; n0 < N; n0 += NB * lanes) {
            if (n0 != nl) {
#pragma unroll
                for (int i = 0; i < NB; i++) {
                    const int n = n0 + i * lanes;
                    if (n < N) s[i] = load_vec<V>(Sg + (int64_t)n * dv);
                }
            }
#pragma unroll
            for (int i = 0; i < NB; i++) {
                const int n = n0 + i * lanes;
                if (n < N) {
                    const float b = bs[n], c = cs[n];
#pragma unroll
                    for (int j = 0; j < V; j++) {
                        s[i].x[j] = fmaf(al, s[i].x[j], b * xv.x[j]);
                        acc.x[j] = fmaf(c, s[i].x[j], acc.x[j]);
                    }
                    store_vec<V>(Sg + (int64_t)n * dv, s[i]);
                }
            }
        }
        store_vec<V>(ps + nl * sl + cg * V, acc);
    }
    __syncthreads();
    float* yr = a.y + (int64_t)t * a.inner + head * dv + slice * sl;
    for (int c = tid; c < sl; c += kThreads) {
        float o = 0.f;
        for (int l = 0; l < lanes; l++) o += ps[l * sl + c];
        yr[c] = fmaf(dskip, xs[c], o) * silu_f(c == tid ? z_first : z[c]);
    }
}

// ---- portions ------------------------------------------------------------------------------------------------

// The request and first row of the step's chunk number `chunk` of KC rows; false beyond the last chunk.
template <int KC>
__device__ __forceinline__ bool find_chunk(const SsdArgs& a, int chunk, int& req, int& row0, int& rows, int& index) {
    for (req = 0; req < a.n_requests; req++) {
        const int lo = a.q_start[req], len = a.q_start[req + 1] - lo, chunks = (len + KC - 1) / KC;
        if (chunk < chunks) {
            index = chunk;
            row0 = lo + chunk * KC;
            rows = min(KC, len - chunk * KC);
            return true;
        }
        chunk -= chunks;
    }
    return false;
}

__device__ __forceinline__ void cp_async16(float* smem, const float* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;                     // 0: the 16 bytes are filled with zeros, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// grid (chunk bound * KC / kRun, blocks of kThreads channels, then blocks of 8 heads).  A thread owns a channel of kRun of the
// chunk's rows; of the further blocks those of a chunk's first run form its decays, one warp per head.  TAPS > 0: that many
// taps, the inputs in registers; 0: any number.
constexpr int kRun = 32;

template <int TAPS, typename T, int KC>
__global__ void __launch_bounds__(kThreads)
conv_kernel(const SsdArgs a) {
    griddep_wait();
    griddep_launch();
    int req, row0, rows, index;
    const int chunk = blockIdx.x / (KC / kRun), run0 = (blockIdx.x % (KC / kRun)) * kRun;
    if (!find_chunk<KC>(a, chunk, req, row0, rows, index)) return;
    const int ch_blocks = (a.channels + kThreads - 1) / kThreads;
    if ((int)blockIdx.y >= ch_blocks) {
        constexpr int R = KC / 32;                          // rows of a lane, one behind the other
        const int h = (blockIdx.y - ch_blocks) * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
        if (run0 > 0 || h >= a.heads) return;
        const float rate = expf(a.a_log[h]), bias = a.dt_bias[h];
        const float* src = a.proj + (int64_t)row0 * a.stride + a.inner + a.channels + h;
        float dt[R];
#pragma unroll
        for (int i = 0; i < R; i++) {
            const int r = lane * R + i;
            dt[i] = r < rows ? src[(int64_t)r * a.stride] : 0.f;
        }
        double part[R], mine = 0.0;
#pragma unroll
        for (int i = 0; i < R; i++) {
            dt[i] = softplus_f(dt[i] + bias);
            mine -= (double)(rate * dt[i]);
            part[i] = mine;
        }
        double sum = mine;                                  // over the lanes up to and including this one
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double other = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += other;
        }
        const double base = sum - mine;
        const int64_t at = ((int64_t)chunk * a.heads + h) * KC + lane * R;
#pragma unroll
        for (int i = 0; i < R; i++) {
            if (lane * R + i < rows) {
                const double v = base + part[i];
                const float hi = (float)v;
                a.dt[at + i] = dt[i];
                a.cum[at + i] = make_float2(hi, (float)(v - (double)hi));
            }
        }
        return;
    }
    const int c = blockIdx.y * kThreads + threadIdx.x, n = min(kRun, rows - run0);
    if (c >= a.channels || n <= 0) return;
    const int taps = TAPS > 0 ? TAPS : a.taps;
    const int first = index * KC + run0;                    // the run's first row, counted from the portion's start
    const float* src = a.proj + (int64_t)(row0 + run0) * a.stride + a.inner + c;
    T* dst = reinterpret_cast<T*>(a.xc) + (int64_t)(row0 + run0) * a.xc_pad + c;
    float* ring = a.ring + (int64_t)a.state_slots[req] * a.ring_stride + c;
    const int p0 = a.start_pos[req] + first;                // position of the run's first row
    const float* w = a.conv_w + (int64_t)c * taps;
    const float bias = a.conv_b[c];
    // input of row r, also in front of the run: an earlier row of the portion, or the ring
    auto input = [&](int r) {
        if (first + r >= 0) return src[(int64_t)r * a.stride];
        const int q = p0 + r;
        return q >= 0 ? ring[(int64_t)(q % taps) * a.ch_pad] : 0.f;
    };
    if constexpr (TAPS > 0) {
        float k[TAPS], u[TAPS];
#pragma unroll
        for (int i = 0; i < TAPS; i++) {
            k[i] = w[i];
            u[i] = i < TAPS - 1 ? input(i - (TAPS - 1)) : 0.f;
        }
        constexpr int AHEAD = 16;
        for (int r0 = 0; r0 < n; r0 += AHEAD) {
            float in[AHEAD];
#pragma unroll
            for (int j = 0; j < AHEAD; j++) in[j] = r0 + j < n ? src[(int64_t)(r0 + j) * a.stride] : 0.f;
#pragma unroll
            for (int j = 0; j < AHEAD; j++) {
                if (r0 + j < n) {
                    u[TAPS - 1] = in[j];
                    float v = bias;
#pragma unroll
                    for (int i = 0; i < TAPS; i++) v = fmaf(k[i], u[i], v);
                    dst[(int64_t)(r0 + j) * a.xc_pad] = from_f32<T>(silu_f(v));
#pragma unroll
                    for (int i = 0; i < TAPS - 1; i++) u[i] = u[i + 1];
                }
            }
        }
    } else {
        for (int r = 0; r < n; r++) {
            float v = bias;
            for (int i = 0; i < taps; i++) v = fmaf(w[i], input(r - (taps - 1) + i), v);
            dst[(int64_t)r * a.xc_pad] = from_f32<T>(silu_f(v));
        }
    }
}

// grid (blocks of kThreads channels, requests), behind conv_kernel: the ring takes the portion's last inputs.
__global__ void __launch_bounds__(kThreads)
ring_kernel(const SsdArgs a) {
    griddep_wait();
    griddep_launch();
    const int c = blockIdx.x * kThreads + threadIdx.x, req = blockIdx.y;
    if (c >= a.channels) return;
    const int lo = a.q_start[req], len = a.q_start[req + 1] - lo;
    float* ring = a.ring + (int64_t)a.state_slots[req] * a.ring_stride + c;
    for (int r = max(0, len - a.taps); r < len; r++)
        ring[(int64_t)((a.start_pos[req] + r) % a.taps) * a.ch_pad] = a.proj[(int64_t)(lo + r) * a.stride + a.inner + c];
}

// grid (chunk bound, groups): pairs[i][j] = C_i . B_j.  Thread (ty, tx): rows 4 ty .., columns 4 tx .. .
// Shared memory: C and B, kKP of their N values at a time, [kKP][kC + 4] each.
constexpr int kKP = 32;

__global__ void __launch_bounds__(kThreads)
pairs_kernel(const SsdArgs a) {
    __shared__ __align__(16) float Cs[kKP][kC + 4], Bs[kKP][kC + 4];
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, group = blockIdx.y, N = a.N;
    int req, row0, rows, index;
    if (!find_chunk<kC>(a, blockIdx.x, req, row0, rows, index)) return;
    const float* B = reinterpret_cast<const float*>(a.xc) + (int64_t)row0 * a.xc_pad + a.inner + group * N;
    const float* C = B + a.groups * N;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < N; k0 += kKP) {
        for (int i = tid; i < kC * kKP; i += kThreads) {
            const int r = i / kKP, k = i - r * kKP;
            const bool in = r < rows && k0 + k < N;
            Cs[k][r] = in ? C[(int64_t)r * a.xc_pad + k0 + k] : 0.f;
            Bs[k][r] = in ? B[(int64_t)r * a.xc_pad + k0 + k] : 0.f;
        }
        __syncthreads();
        if (tx <= ty) {                                      // blocks of four that hold a pair j <= i
#pragma unroll 8
            for (int k = 0; k < kKP; k++) {
                const float4 c4 = *reinterpret_cast<const float4*>(&Cs[k][4 * ty]);
                const float4 b4 = *reinterpret_cast<const float4*>(&Bs[k][4 * tx]);
                const float c[4] = {c4.x, c4.y, c4.z, c4.w}, b[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[i][j] = fmaf(c[i], b[j], acc[i][j]);
            }
        }
        __syncthreads();
    }
    float* out = a.pairs + ((int64_t)blockIdx.x * a.groups + group) * kC * kC;
#pragma unroll
    for (int i = 0; i < 4; i++)
        *reinterpret_cast<float4*>(out + (4 * ty + i) * kC + 4 * tx) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}

// N consecutive values of shared memory as the register tile of thread `t` of 16: fours at 64 u + 4 t (N 4, 8), or two at 2 t
template <int N> __device__ __forceinline__ int tile_at(int t, int i) { return N == 2 ? 2 * t + i : (i >> 2) * 64 + 4 * t + (i & 3); }

// grid (chunk bound, heads, tiles of 16 RM state channels by 16 RN value channels): s_in = sum over the chunk's rows of
// exp(c_last - c_j) dt_j B_j x_j^T.  Thread (ty, tx): an RM x RN tile.  Shared memory: B [kC][16 RM], x [kC][16 RN], weights [kC].
template <int RM, int RN>
__global__ void __launch_bounds__(kThreads)
outer_kernel(const SsdArgs a, int e_tiles) {
    extern __shared__ __align__(16) float sm[];
    constexpr int TM = 16 * RM, TN = 16 * RN;
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int head = blockIdx.y, d0 = blockIdx.z / e_tiles * TM, e0 = blockIdx.z % e_tiles * TN, N = a.N, dv = a.dv;
    int req, row0, rows, index;
    if (!find_chunk<kC>(a, blockIdx.x, req, row0, rows, index)) return;
    float* ks = sm;
    float* vs = ks + kC * TM;
    float* ws = vs + kC * TN;
    const float* kg = reinterpret_cast<const float*>(a.xc) + (int64_t)row0 * a.xc_pad + a.inner + (head / (a.heads / a.groups)) * N + d0;
    const float* vg = reinterpret_cast<const float*>(a.xc) + (int64_t)row0 * a.xc_pad + head * dv + e0;
    if (a.vec) {
        for (int i = tid; i < rows * (TM / 4); i += kThreads) {
            const int r = i / (TM / 4), d = (i - r * (TM / 4)) * 4;
            cp_async16(ks + r * TM + d, kg + (d0 + d < N ? (int64_t)r * a.xc_pad + d : 0), d0 + d < N);
        }
        for (int i = tid; i < rows * (TN / 4); i += kThreads) {
            const int r = i / (TN / 4), c = (i - r * (TN / 4)) * 4;
            cp_async16(vs + r * TN + c, vg + (e0 + c < dv ? (int64_t)r * a.xc_pad + c : 0), e0 + c < dv);
        }
        cp_async_commit();
    } else {
        for (int i = tid; i < rows * TM; i += kThreads) {
            const int r = i / TM, d = i - r * TM;
            ks[i] = d0 + d < N ? kg[(int64_t)r * a.xc_pad + d] : 0.f;
        }
        for (int i = tid; i < rows * TN; i += kThreads) {
            const int r = i / TN, c = i - r * TN;
            vs[i] = e0 + c < dv ? vg[(int64_t)r * a.xc_pad + c] : 0.f;
        }
    }
    if (tid < rows) {
        const int64_t at = ((int64_t)blockIdx.x * a.heads + head) * kC;
        ws[tid] = exp_diff(a.cum[at + rows - 1], a.cum[at + tid]) * a.dt[at + tid];
    }
    cp_async_wait<0>();
    __syncthreads();
    float acc[RM][RN];
#pragma unroll
    for (int m = 0; m < RM; m++)
#pragma unroll
        for (int n = 0; n < RN; n++) acc[m][n] = 0.f;
#pragma unroll 2
    for (int r = 0; r < rows; r++) {
        float k[RM], v[RN];
        const float w = ws[r];
        if constexpr (RM == 2) {
            const float2 t = *reinterpret_cast<const float2*>(ks + r * TM + 2 * ty);
            k[0] = t.x; k[1] = t.y;
        } else {
#pragma unroll
            for (int u = 0; u < RM / 4; u++) {
                const float4 t = *reinterpret_cast<const float4*>(ks + r * TM + u * 64 + 4 * ty);
                k[4 * u] = t.x; k[4 * u + 1] = t.y; k[4 * u + 2] = t.z; k[4 * u + 3] = t.w;
            }
        }
#pragma unroll
        for (int u = 0; u < RN / 4; u++) {
            const float4 t = *reinterpret_cast<const float4*>(vs + r * TN + u * 64 + 4 * tx);
            v[4 * u] = t.x * w; v[4 * u + 1] = t.y * w; v[4 * u + 2] = t.z * w; v[4 * u + 3] = t.w * w;
        }
#pragma unroll
        for (int m = 0; m < RM; m++)
#pragma unroll
            for (int n = 0; n < RN; n++) acc[m][n] = fmaf(k[m], v[n], acc[m][n]);
    }
    float* S = a.s_in + ((int64_t)blockIdx.x * a.heads + head) * N * dv;
#pragma unroll
    for (int m = 0; m < RM; m++) {
        const int d = d0 + tile_at<RM>(ty, m);
        if (d >= N) continue;
#pragma unroll
        for (int u = 0; u < RN / 4; u++) {
            const int e = e0 + u * 64 + 4 * tx;
            if (a.vec) {
                if (e < dv)
                    *reinterpret_cast<float4*>(S + (int64_t)d * dv + e) =
                        make_float4(acc[m][4 * u], acc[m][4 * u + 1], acc[m][4 * u + 2], acc[m][4 * u + 3]);
            } else {
#pragma unroll
                for (int i = 0; i < 4; i++)
                    if (e + i < dv) S[(int64_t)d * dv + e + i] = acc[m][4 * u + i];
            }
        }
    }
}

// grid (pieces of kThreads * V state elements, heads, requests): s_in turns from the chunks' own states into the
// states at their starts; SPLIT: those go to s_split.
template <int V, int KC, bool SPLIT>
__global__ void __launch_bounds__(kThreads)
carry_kernel(const SsdArgs a) {
    griddep_wait();
    griddep_launch();
    const int head = blockIdx.y, req = blockIdx.z;
    const int64_t elems = (int64_t)a.N * a.dv, i = ((int64_t)blockIdx.x * kThreads + threadIdx.x) * V;
    if (i >= elems) return;
    int chunk = 0;
    for (int r = 0; r < req; r++) chunk += (a.q_start[r + 1] - a.q_start[r] + KC - 1) / KC;
    const int len = a.q_start[req + 1] - a.q_start[req], chunks = (len + KC - 1) / KC;
    float* slot = a.state + (int64_t)a.state_slots[req] * a.state_stride + head * elems + i;
    float* w = a.s_in + ((int64_t)chunk * a.heads + head) * elems + i;
    const float2* cum = a.cum + ((int64_t)chunk * a.heads + head) * KC;
    const int64_t step = a.heads * elems, cum_step = (int64_t)a.heads * KC;
    Vec<V> s = load_vec<V>(slot);
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        Vec<V> loc[AHEAD];
        float d[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                loc[u] = load_vec<V>(w + (c0 + u) * step);
                const float2 last = cum[(c0 + u) * cum_step + min(KC, len - (c0 + u) * KC) - 1];
                d[u] = expf(last.x + last.y);
            }
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                if constexpr (SPLIT) {
                    bf16 hi[V], lo[V];
#pragma unroll
                    for (int j = 0; j < V; j++) {
                        hi[j] = __float2bfloat16_rn(s.x[j]);
                        lo[j] = __float2bfloat16_rn(s.x[j] - __bfloat162float(hi[j]));
                    }
                    bf16* dst = a.s_split + (w - a.s_in) + (c0 + u) * step;
                    static_assert(V == 4, "eight bytes at a time");
                    *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(hi);
                    *reinterpret_cast<uint2*>(dst + a.split_plane) = *reinterpret_cast<const uint2*>(lo);
                } else {
                    store_vec<V>(w + (c0 + u) * step, s);
                }
#pragma unroll
                for (int j = 0; j < V; j++) s.x[j] = fmaf(d[u], s.x[j], loc[u].x[j]);
            }
    }
    store_vec<V>(slot, s);
}

// grid (chunk bound, heads, column blocks of 64 NJ): [exp(c) C | weights] [S_in ; x], in blocks of kKB inner elements, two of
// them in shared memory.  Thread (rg, cg): rows 4 rg .. 4 rg + 3, value channels j * 64 + 4 cg .. + 3.
// Shared memory, twice: left [kC][kKB + 4], right [kKB][64 NJ]; then the chunk's sums and steps [kC] each.
constexpr int kKB = 32;

template <int NJ>
__global__ void __launch_bounds__(kThreads)
apply_kernel(const SsdArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int QP = kKB + 4, CW = 64 * NJ, STAGE = kC * QP + kKB * CW;
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, cg = tid & 15, rg = tid >> 4;
    const int head = blockIdx.y, e0 = blockIdx.z * CW, N = a.N, dv = a.dv, group = head / (a.heads / a.groups);
    const int ne = min(CW, dv - e0);
    int req, row0, rows, index;
    if (!find_chunk<kC>(a, blockIdx.x, req, row0, rows, index)) return;
    float2* cum = reinterpret_cast<float2*>(sm + 2 * STAGE);
    float* dts = reinterpret_cast<float*>(cum + kC);
    if (tid < kC) {
        const int64_t at = ((int64_t)blockIdx.x * a.heads + head) * kC + min(tid, rows - 1);
        cum[tid] = a.cum[at];
        dts[tid] = a.dt[at];
    }
    float acc[4][NJ * 4];
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int j = 0; j < NJ * 4; j++) acc[r][j] = 0.f;
    const bool from_zero = index == 0 && a.start_pos[req] == 0;        // the state in front of a request's first chunk
    const int nb_s = from_zero ? 0 : (N + kKB - 1) / kKB, nb = nb_s + (rows + kKB - 1) / kKB;
    const float* S = a.s_in + ((int64_t)blockIdx.x * a.heads + head) * N * dv + e0;
    const float* W = a.pairs + ((int64_t)blockIdx.x * a.groups + group) * kC * kC;
    const float* xg = reinterpret_cast<const float*>(a.xc) + (int64_t)row0 * a.xc_pad + head * dv + e0;
    const float* Cg = reinterpret_cast<const float*>(a.xc) + (int64_t)row0 * a.xc_pad + a.inner + (a.groups + group) * N;
    auto load = [&](int b) {                // inner elements k0 .. k0 + kKB - 1 of the state's part, then of the chunk's own
        float* left = sm + (b & 1) * STAGE;
        float* right = left + kC * QP;
        const bool state = b < nb_s;
        const int k0 = (state ? b : b - nb_s) * kKB, nk = min(kKB, (state ? N : rows) - k0);
        const float* lg = state ? Cg + k0 : W + k0;
        const float* rg_ = state ? S + (int64_t)k0 * dv : xg + (int64_t)k0 * a.xc_pad;
        const int64_t ls = state ? a.xc_pad : kC, rs = state ? dv : a.xc_pad;
        if (a.vec) {
            for (int i = tid; i < kC * (kKB / 4); i += kThreads) {
                const int r = i / (kKB / 4), k = (i - r * (kKB / 4)) * 4;
                const bool in = r < rows && (state ? k < nk : true);      // the pairs' rows are whole
                cp_async16(left + r * QP + k, lg + (in ? r * ls + k : 0), in);
            }
            for (int i = tid; i < kKB * (CW / 4); i += kThreads) {
                const int k = i / (CW / 4), c = (i - k * (CW / 4)) * 4;
                const bool in = k < nk && c < ne;
                cp_async16(right + k * CW + c, rg_ + (in ? k * rs + c : 0), in);
            }
        } else {
            for (int i = tid; i < kC * kKB; i += kThreads) {
                const int r = i / kKB, k = i - r * kKB;
                left[r * QP + k] = (r < rows && k < nk) ? lg[r * ls + k] : 0.f;
            }
            for (int i = tid; i < kKB * CW; i += kThreads) {
                const int k = i / CW, c = i - k * CW;
                right[i] = (k < nk && c < ne) ? rg_[k * rs + c] : 0.f;
            }
        }
        cp_async_commit();
    };
    load(0);
    for (int b = 0; b < nb; b++) {
        if (b + 1 < nb) {
            load(b + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        float* qs = sm + (b & 1) * STAGE;
        const float* ss = qs + kC * QP;
        // the left block's decays, in place: a pair's, or the row's own towards the state
        const bool state = b < nb_s;
        const int k0 = state ? 0 : (b - nb_s) * kKB;
        for (int i = tid; i < kC * kKB; i += kThreads) {
            const int r = i / kKB, k = i - r * kKB, j = k0 + k;
            float f;
            if (state) f = expf(cum[r].x + cum[r].y);
            else f = j <= r && r < rows ? exp_diff(cum[r], cum[j]) * dts[j] : 0.f;
            qs[r * QP + k] = f == 0.f ? 0.f : qs[r * QP + k] * f;
        }
        __syncthreads();
#pragma unroll 2
        for (int d = 0; d < kKB; d += 4) {
            float q[4][4];
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const float4 q4 = *reinterpret_cast<const float4*>(qs + (rg * 4 + r) * QP + d);
                q[r][0] = q4.x; q[r][1] = q4.y; q[r][2] = q4.z; q[r][3] = q4.w;
            }
#pragma unroll
            for (int j = 0; j < NJ; j++)
#pragma unroll
                for (int u = 0; u < 4; u++) {
                    const float4 s4 = *reinterpret_cast<const float4*>(ss + (d + u) * CW + j * 64 + cg * 4);
#pragma unroll
                    for (int r = 0; r < 4; r++) {
                        acc[r][j * 4 + 0] = fmaf(q[r][u], s4.x, acc[r][j * 4 + 0]);
                        acc[r][j * 4 + 1] = fmaf(q[r][u], s4.y, acc[r][j * 4 + 1]);
                        acc[r][j * 4 + 2] = fmaf(q[r][u], s4.z, acc[r][j * 4 + 2]);
                        acc[r][j * 4 + 3] = fmaf(q[r][u], s4.w, acc[r][j * 4 + 3]);
                    }
                }
        }
        __syncthreads();                    // this stage may be loaded again
    }
    const float dskip = a.d[head];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int row = rg * 4 + r;
        if (row >= rows) continue;
        const float* xr = xg + (int64_t)row * a.xc_pad;
        const float* zr = a.proj + (int64_t)(row0 + row) * a.stride + head * dv + e0;
        float* yr = a.y + (int64_t)(row0 + row) * a.inner + head * dv + e0;
#pragma unroll
        for (int j = 0; j < NJ; j++) {
            const int col = j * 64 + cg * 4;
            if (a.vec) {
                if (col >= ne) continue;
                const float4 x4 = *reinterpret_cast<const float4*>(xr + col), z4 = *reinterpret_cast<const float4*>(zr + col);
                *reinterpret_cast<float4*>(yr + col) =
                    make_float4(fmaf(dskip, x4.x, acc[r][j * 4]) * silu_f(z4.x), fmaf(dskip, x4.y, acc[r][j * 4 + 1]) * silu_f(z4.y),
                                fmaf(dskip, x4.z, acc[r][j * 4 + 2]) * silu_f(z4.z), fmaf(dskip, x4.w, acc[r][j * 4 + 3]) * silu_f(z4.w));
            } else {
#pragma unroll
                for (int c = 0; c < 4; c++)
                    if (col + c < ne) yr[col + c] = fmaf(dskip, xr[col + c], acc[r][j * 4 + c]) * silu_f(zr[col + c]);
            }
        }
    }
}

// ---- portions in bfloat16 on the tensor cores -------------------------------------------------------------------

__device__ __forceinline__ void cp16(bf16* smem, const bf16* gmem, bool valid) {
    cp_async16(reinterpret_cast<float*>(smem), reinterpret_cast<const float*>(gmem), valid);
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], const bf16* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two values as a pair of bfloat16, and what that rounding left as another
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

constexpr int kDB = 64;                     // value channels of a CTA
constexpr int kXP = kDB + 8;                // padded row of such a block, in elements

// Fragments of rows k0 .. k0 + 15 of a block at row length kXP, as the second operand: b[p] for columns 16 p .. 16 p + 15.  All
// loads go out before the first product that needs one.
__device__ __forceinline__ void load_block(uint32_t (&b)[4][4], const bf16* block, int k0, int lane) {
    const int mi = lane >> 3;
    const bf16* base = block + (k0 + (mi & 1) * 8 + (lane & 7)) * kXP + (mi >> 1) * 8;
#pragma unroll
    for (int p = 0; p < kDB / 16; p++) ldsm4_trans(b[p], base + p * 16);
}
__device__ __forceinline__ void times_block(float (&acc)[8][4], const uint32_t (&a)[4], const uint32_t (&b)[4][4]) {
#pragma unroll
    for (int p = 0; p < kDB / 16; p++) {
        mma16816(acc[2 * p], a, b[p][0], b[p][1]);
        mma16816(acc[2 * p + 1], a, b[p][2], b[p][3]);
    }
}

// grid (chunk bound, heads, blocks of kDB value channels): s_in = sum over the chunk's rows of exp(c_last - c_j) dt_j B_j x_j^T.
// Warp w: state channels 16 w .., 16 (w + 8) .., ...  Shared memory: B [kT][N + 8], the weighted rows [kT][kXP] high and low, weights [kT].
__global__ void __launch_bounds__(kThreads)
outer_tc_kernel(const SsdArgs a) {
    extern __shared__ __align__(16) float sm[];
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tq = lane & 3, mi = lane >> 3;
    const int head = blockIdx.y, e0 = blockIdx.z * kDB, N = a.N, dv = a.dv, NP = N + 8, ne = min(kDB, dv - e0);
    int req, row0, rows, index;
    if (!find_chunk<kT>(a, blockIdx.x, req, row0, rows, index)) return;
    bf16* Bs = reinterpret_cast<bf16*>(sm);
    bf16* xh = Bs + kT * NP;
    bf16* xl = xh + kT * kXP;
    float* ws = reinterpret_cast<float*>(xl + kT * kXP);
    const bf16* xg = reinterpret_cast<const bf16*>(a.xc) + (int64_t)row0 * a.xc_pad;
    const bf16* bg = xg + a.inner + (head / (a.heads / a.groups)) * N;
    const int steps = (rows + 15) / 16, per = N / 8;
    for (int i = tid; i < steps * 16 * per; i += kThreads) {
        const int r = i / per, c = (i - r * per) * 8;
        cp16(Bs + r * NP + c, bg + (r < rows ? (int64_t)r * a.xc_pad + c : 0), r < rows);
    }
    cp_async_commit();
    if (tid < kT) {
        const int64_t at = ((int64_t)blockIdx.x * a.heads + head) * kT;
        ws[tid] = tid < rows ? exp_diff(a.cum[at + rows - 1], a.cum[at + tid]) * a.dt[at + tid] : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < steps * 16 * (kDB / 8); i += kThreads) {
        const int r = i / (kDB / 8), c = (i - r * (kDB / 8)) * 8;
        uint4 h = make_uint4(0, 0, 0, 0), l = h;
        if (r < rows && c < ne) {
            const uint4 v = *reinterpret_cast<const uint4*>(xg + (int64_t)r * a.xc_pad + head * dv + e0 + c);
            const float w = ws[r];
            auto part = [&](uint32_t in, uint32_t& hi, uint32_t& lo) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in));
                split2(f.x * w, f.y * w, hi, lo);
            };
            part(v.x, h.x, l.x); part(v.y, h.y, l.y); part(v.z, h.z, l.z); part(v.w, h.w, l.w);
        }
        *reinterpret_cast<uint4*>(xh + r * kXP + c) = h;
        *reinterpret_cast<uint4*>(xl + r * kXP + c) = l;
    }
    cp_async_wait<0>();
    __syncthreads();
    float* S = a.s_in + ((int64_t)blockIdx.x * a.heads + head) * N * dv + e0;
    for (int m0 = warp * 16; m0 < N; m0 += 16 * (kThreads / 32)) {
        float acc[8][4];
#pragma unroll
        for (int i = 0; i < 8; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
        for (int k = 0; k < steps; k++) {
            uint32_t af[4];
            ldsm4_trans(af, Bs + (k * 16 + (mi >> 1) * 8 + (lane & 7)) * NP + m0 + (mi & 1) * 8);
            uint32_t bh[4][4], bl[4][4];
            load_block(bh, xh, k * 16, lane);
            load_block(bl, xl, k * 16, lane);
            times_block(acc, af, bh);
            times_block(acc, af, bl);
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int c = i * 8 + 2 * tq;
            if (c >= ne) continue;
            *reinterpret_cast<float2*>(S + (int64_t)(m0 + gid) * dv + c) = make_float2(acc[i][0], acc[i][1]);
            *reinterpret_cast<float2*>(S + (int64_t)(m0 + gid + 8) * dv + c) = make_float2(acc[i][2], acc[i][3]);
        }
    }
}

// grid (chunk bound, heads, blocks of kDB value channels).  Warp w: rows 16 w .. 16 w + 15 of the chunk.
// Shared memory: C [kT][N + 8]; the state's two terms [N][kXP] each, then B [kT][N + 8] in their place; x [kT][kXP]; sums and steps [kT].
__global__ void __launch_bounds__(kThreads, 2)
apply_tc_kernel(const SsdArgs a, int shared_place) {
    extern __shared__ __align__(16) float sm[];
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tq = lane & 3, mi = lane >> 3;
    const int head = blockIdx.y, e0 = blockIdx.z * kDB, N = a.N, dv = a.dv, NP = N + 8, ne = min(kDB, dv - e0);
    const int group = head / (a.heads / a.groups), per = N / 8;
    int req, row0, rows, index;
    if (!find_chunk<kT>(a, blockIdx.x, req, row0, rows, index)) return;
    bf16* Cs = reinterpret_cast<bf16*>(sm);
    bf16* Us = Cs + kT * NP;
    bf16* xs = Us + shared_place;
    float2* cum = reinterpret_cast<float2*>(xs + kT * kXP);
    float* dts = reinterpret_cast<float*>(cum + kT);
    const bf16* xg = reinterpret_cast<const bf16*>(a.xc) + (int64_t)row0 * a.xc_pad;
    const bf16* bg = xg + a.inner + group * N;
    const bf16* cg = bg + a.groups * N;
    const int rows16 = (rows + 15) / 16 * 16;
    const bool from_zero = index == 0 && a.start_pos[req] == 0;        // the state in front of a request's first chunk
    for (int i = tid; i < rows16 * per; i += kThreads) {
        const int r = i / per, c = (i - r * per) * 8;
        cp16(Cs + r * NP + c, cg + (r < rows ? (int64_t)r * a.xc_pad + c : 0), r < rows);
    }
    auto load_b = [&]() {
        for (int i = tid; i < rows16 * per; i += kThreads) {
            const int r = i / per, c = (i - r * per) * 8;
            cp16(Us + r * NP + c, bg + (r < rows ? (int64_t)r * a.xc_pad + c : 0), r < rows);
        }
    };
    if (from_zero) {
        load_b();
    } else {
        const bf16* S = a.s_split + ((int64_t)blockIdx.x * a.heads + head) * N * dv + e0;
        for (int i = tid; i < 2 * N * (kDB / 8); i += kThreads) {
            const int r = i / (kDB / 8), c = (i - r * (kDB / 8)) * 8, n = r < N ? r : r - N;
            const bool in = c < ne;
            cp16(Us + r * kXP + c, S + (in ? (r < N ? 0 : a.split_plane) + (int64_t)n * dv + c : 0), in);
        }
    }
    for (int i = tid; i < rows16 * (kDB / 8); i += kThreads) {
        const int r = i / (kDB / 8), c = (i - r * (kDB / 8)) * 8;
        const bool in = r < rows && c < ne;
        cp16(xs + r * kXP + c, xg + (in ? (int64_t)r * a.xc_pad + head * dv + e0 + c : 0), in);
    }
    cp_async_commit();
    if (tid < kT) {
        const int64_t at = ((int64_t)blockIdx.x * a.heads + head) * kT + min(tid, rows - 1);
        cum[tid] = a.cum[at];
        dts[tid] = a.dt[at];
    }
    cp_async_wait<0>();
    __syncthreads();
    const bool active = 16 * warp < rows;
    const bf16* ca = Cs + (16 * warp + (lane & 15)) * NP + (lane >> 4) * 8;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    const int i0 = 16 * warp + gid, i1 = i0 + 8;
    const float2 ci0 = cum[min(i0, kT - 1)], ci1 = cum[min(i1, kT - 1)];
    if (!from_zero) {
        if (active) {
            for (int k = 0; k < N; k += 16) {
                uint32_t af[4];
                ldsm4(af, ca + k);
                uint32_t bh[4][4], bl[4][4];
                load_block(bh, Us, k, lane);
                load_block(bl, Us + N * kXP, k, lane);
                times_block(acc, af, bh);
                times_block(acc, af, bl);
            }
            const float f0 = expf(ci0.x + ci0.y), f1 = expf(ci1.x + ci1.y);
#pragma unroll
            for (int i = 0; i < 8; i++) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
        }
        __syncthreads();                    // the state's place takes B
        load_b();
        cp_async_commit();
        cp_async_wait<0>();
        __syncthreads();
    }
    if (!active) return;
    for (int key0 = 0; key0 <= 16 * warp; key0 += 64) {
        const int slices = min(4, (16 * warp - key0) / 16 + 1);          // slices of 16 keys that hold a pair j <= i
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) s[i][j] = 0.f;
        const bf16* kb = Us + (key0 + (mi >> 1) * 8 + (lane & 7)) * NP + (mi & 1) * 8;
        for (int k = 0; k < N; k += 16) {
            uint32_t af[4], b[4][4];
            ldsm4(af, ca + k);
#pragma unroll
            for (int sl = 0; sl < 4; sl++)
                if (sl < slices) ldsm4(b[sl], kb + 16 * sl * NP + k);
#pragma unroll
            for (int sl = 0; sl < 4; sl++) {
                if (sl < slices) {
                    mma16816(s[2 * sl], af, b[sl][0], b[sl][1]);
                    mma16816(s[2 * sl + 1], af, b[sl][2], b[sl][3]);
                }
            }
        }
#pragma unroll
        for (int sl = 0; sl < 4; sl++) {
            if (sl < slices) {
                uint32_t ph[4], pl[4], xb[4][4];
                load_block(xb, xs, key0 + 16 * sl, lane);
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    float p[4];
#pragma unroll
                    for (int u = 0; u < 2; u++) {
                        const int j = key0 + 16 * sl + 8 * h + 2 * tq + u;
                        const float2 cj = cum[j];
                        const float d = dts[j];
                        p[u] = j <= i0 ? s[2 * sl + h][u] * (exp_diff(ci0, cj) * d) : 0.f;
                        p[2 + u] = j <= i1 ? s[2 * sl + h][2 + u] * (exp_diff(ci1, cj) * d) : 0.f;
                    }
                    split2(p[0], p[1], ph[2 * h], pl[2 * h]);
                    split2(p[2], p[3], ph[2 * h + 1], pl[2 * h + 1]);
                }
                times_block(acc, ph, xb);
                times_block(acc, pl, xb);
            }
        }
    }
    const float dskip = a.d[head];
    float2 zv[2][8];                        // all of the gate's loads before the first store
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const float* zr = a.proj + (int64_t)(row0 + min(h ? i1 : i0, rows - 1)) * a.stride + head * dv + e0;
#pragma unroll
        for (int i = 0; i < 8; i++) zv[h][i] = *reinterpret_cast<const float2*>(zr + min(i * 8 + 2 * tq, ne - 2));
    }
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int r = h ? i1 : i0;
        if (r >= rows) continue;
        float* yr = a.y + (int64_t)(row0 + r) * a.inner + head * dv + e0;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int c = i * 8 + 2 * tq;
            if (c >= ne) continue;
            const float2 z = zv[h][i];
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(xs + r * kXP + c));
            *reinterpret_cast<float2*>(yr + c) =
                make_float2(fmaf(dskip, x.x, acc[i][2 * h]) * silu_f(z.x), fmaf(dskip, x.y, acc[i][2 * h + 1]) * silu_f(z.y));
        }
    }
}

// out[r][part] = y[r][part] / rms(y[r][part]) * gain of w values.  WARP: one warp per (row, part), eight to a CTA; else one
// CTA.  VEC: w a multiple of 4 up to 4 * kVec * (threads of a part), 16-byte rows, the values in registers between the
// sum and the scaling.
constexpr int kVec = 8;

template <typename T, bool VEC, bool WARP>
__global__ void __launch_bounds__(kThreads)
part_norm_kernel(T* __restrict__ out, int64_t out_stride, const float* __restrict__ y, const float* __restrict__ gain, int parts,
                 int w, float eps, int64_t items) {
    __shared__ float red[32];
    griddep_wait();
    griddep_launch();
    const int64_t item = WARP ? (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5) : blockIdx.x;
    if (item >= items) return;
    const int me = WARP ? threadIdx.x & 31 : threadIdx.x, all = WARP ? 32 : blockDim.x;
    const int64_t r = item / parts;
    const int part = (int)(item - r * parts);
    const float* src = y + item * w;
    const float* g = gain + (int64_t)part * w;
    T* dst = out + r * out_stride + (int64_t)part * w;
    float sq = 0.f;
    auto total = [&](float v) {
        if constexpr (WARP) return warp_sum(v);
        else return block_sum(v, red);
    };
    if constexpr (VEC) {
        const int w4 = w >> 2;
        float4 v[kVec];
#pragma unroll
        for (int k = 0; k < kVec; k++) {
            const int i = me + k * all;
            if (i < w4) {
                v[k] = reinterpret_cast<const float4*>(src)[i];
                sq += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
            }
        }
        const float scale = rsqrtf(total(sq) / (float)w + eps);
#pragma unroll
        for (int k = 0; k < kVec; k++) {
            const int i = me + k * all;
            if (i < w4) {
                const float4 n4 = reinterpret_cast<const float4*>(g)[i];
                const float o0 = v[k].x * scale * n4.x, o1 = v[k].y * scale * n4.y, o2 = v[k].z * scale * n4.z, o3 = v[k].w * scale * n4.w;
                if constexpr (sizeof(T) == 4) {
                    reinterpret_cast<float4*>(dst)[i] = make_float4(o0, o1, o2, o3);
                } else {
                    __nv_bfloat162 lo = __floats2bfloat162_rn(o0, o1), hi = __floats2bfloat162_rn(o2, o3);
                    uint2 pk;
                    pk.x = *reinterpret_cast<uint32_t*>(&lo);
                    pk.y = *reinterpret_cast<uint32_t*>(&hi);
                    reinterpret_cast<uint2*>(dst)[i] = pk;
                }
            }
        }
    } else {
        for (int i = me; i < w; i += all) sq += src[i] * src[i];
        const float scale = rsqrtf(total(sq) / (float)w + eps);
        for (int i = me; i < w; i += all) dst[i] = from_f32<T>(src[i] * scale * g[i]);
    }
}

template <int V>
int launch_step(const SsdArgs& a, bool early, cudaStream_t s) {
    // slices: a power of two, more of them while the launch would leave SMs idle
    int slices = 1;
    auto splits = [&](int n) { return a.dv % (n * V) == 0; };
    while (a.dv / slices / V > kThreads && splits(slices * 2)) slices *= 2;
    while (splits(slices * 2) && a.dv / (slices * 2) >= 16 && (int64_t)slices * a.heads * a.n_requests < 148) slices *= 2;
    const int sl = a.dv / slices;
    if (sl / V > kThreads) KLLM_FAIL("ssd step: a head of %d value channels does not fit", a.dv);
    const size_t smem = sizeof(float) * ((size_t)kThreads * V + sl + 2 * (size_t)a.N);
    if (smem > 200 * 1024) KLLM_FAIL("ssd step: a state of %d channels does not fit shared memory", a.N);
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(step_kernel<V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) KLLM_FAIL("ssd step: %s", cudaGetErrorString(e));
        raised = true;
    }
    kllm_launch_dep(early, (step_kernel<V>), dim3(slices, a.heads, a.n_requests), dim3(kThreads), smem, s, a, sl);
    KLLM_LAUNCH_STATUS();
}

template <typename K>
int raise_smem(K kern, bool& raised) {
    if (raised) return 0;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) KLLM_FAIL("ssd: %s", cudaGetErrorString(e));
    raised = true;
    return 0;
}

template <int RM, int RN>
int launch_outer(const SsdArgs& a, int chunk_bound, cudaStream_t s) {
    const int e_tiles = (a.dv + 16 * RN - 1) / (16 * RN), d_tiles = (a.N + 16 * RM - 1) / (16 * RM);
    static bool raised = false;
    int rc = raise_smem(outer_kernel<RM, RN>, raised);
    if (rc) return rc;
    kllm_launch((outer_kernel<RM, RN>), dim3(chunk_bound, a.heads, e_tiles * d_tiles), dim3(kThreads),
                sizeof(float) * kC * (16 * (RM + RN) + 1), s, a, e_tiles);
    KLLM_LAUNCH_STATUS();
}

template <int NJ>
int launch_apply(const SsdArgs& a, int chunk_bound, cudaStream_t s) {
    const size_t smem = sizeof(float) * (2 * (kC * (kKB + 4) + kKB * 64 * NJ) + 3 * kC);
    static bool raised = false;
    int rc = raise_smem(apply_kernel<NJ>, raised);
    if (rc) return rc;
    kllm_launch((apply_kernel<NJ>), dim3(chunk_bound, a.heads, (a.dv + 64 * NJ - 1) / (64 * NJ)), dim3(kThreads), smem, s, a);
    KLLM_LAUNCH_STATUS();
}

template <typename T, int KC>
void launch_conv(const SsdArgs& a, int chunk_bound, cudaStream_t s) {
    const int blocks = (a.channels + kThreads - 1) / kThreads;
    const dim3 grid(chunk_bound * (KC / kRun), blocks + (a.heads * 32 + kThreads - 1) / kThreads);
    if (a.taps == 4) kllm_launch((conv_kernel<4, T, KC>), grid, dim3(kThreads), 0, s, a);
    else kllm_launch((conv_kernel<0, T, KC>), grid, dim3(kThreads), 0, s, a);
    kllm_launch((ring_kernel), dim3(blocks, a.n_requests), dim3(kThreads), 0, s, a);
}

template <int V, int KC, bool SPLIT>
void launch_carry(const SsdArgs& a, cudaStream_t s) {
    const int64_t elems = (int64_t)a.N * a.dv;
    kllm_launch((carry_kernel<V, KC, SPLIT>), dim3((unsigned)((elems / V + kThreads - 1) / kThreads), a.heads, a.n_requests), dim3(kThreads), 0,
                s, a);
}

int run_portions(const SsdArgs& a, int chunk_bound, cudaStream_t s) {
    launch_conv<float, kC>(a, chunk_bound, s);
    kllm_launch((pairs_kernel), dim3(chunk_bound, a.groups), dim3(kThreads), 0, s, a);
    int rc;
    if (a.N <= 32) rc = a.dv <= 64 ? launch_outer<2, 4>(a, chunk_bound, s) : launch_outer<2, 8>(a, chunk_bound, s);
    else if (a.N <= 64) rc = a.dv <= 64 ? launch_outer<4, 4>(a, chunk_bound, s) : launch_outer<4, 8>(a, chunk_bound, s);
    else rc = a.dv <= 64 ? launch_outer<8, 4>(a, chunk_bound, s) : launch_outer<8, 8>(a, chunk_bound, s);
    if (rc) return rc;
    if (a.vec) launch_carry<4, kC, false>(a, s);
    else launch_carry<1, kC, false>(a, s);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) KLLM_FAIL("ssd: %s", cudaGetErrorString(e));
    return a.dv <= 64 ? launch_apply<1>(a, chunk_bound, s) : launch_apply<2>(a, chunk_bound, s);
}

int run_portions_tc(const SsdArgs& a, int chunk_bound, cudaStream_t s) {
    const int place = max(2 * a.N * kXP, kT * (a.N + 8));              // elements that the state's terms and B share
    const size_t outer_bytes = sizeof(bf16) * (size_t)kT * (a.N + 8 + 2 * kXP) + sizeof(float) * kT;
    const size_t apply_bytes = sizeof(bf16) * ((size_t)kT * (a.N + 8 + kXP) + place) + 3 * sizeof(float) * kT;
    static bool raised_outer = false, raised_apply = false;
    int rc = raise_smem(outer_tc_kernel, raised_outer);
    if (!rc) rc = raise_smem(apply_tc_kernel, raised_apply);
    if (rc) return rc;
    const dim3 grid(chunk_bound, a.heads, (a.dv + kDB - 1) / kDB);
    launch_conv<bf16, kT>(a, chunk_bound, s);
    kllm_launch((outer_tc_kernel), grid, dim3(kThreads), outer_bytes, s, a);
    launch_carry<4, kT, true>(a, s);
    kllm_launch((apply_tc_kernel), grid, dim3(kThreads), apply_bytes, s, a, place);
    KLLM_LAUNCH_STATUS();
}

// bfloat16 models whose sizes the tensor-core form takes (its shared memory bounds N)
bool tensor_cores(int dtype, int N, int dv) { return dtype == KLLM_BF16 && N % 16 == 0 && dv % 16 == 0 && N <= 256; }

}  // namespace

// Rows of a chunk of the form for portions that these sizes take; kT of the tensor-core form.
extern "C" int kllm_ssd_chunk_rows(int N, int dv, int dtype) { return tensor_cores(dtype, N, dv) ? kT : kC; }

// proj float32 [n] rows at row stride `stride`: z, x (heads * dv each), B, C (groups * N each), dt (heads); conv_w float32
// [channels][taps], conv_b [channels] over x, B and C; dt_bias, a_log, d float32 [heads]; state float32 [slots][state_stride] whose
// first heads * N * dv values are S as [heads][N][dv]; ring float32 [slots][ring_stride] with taps rows of the channels rounded
// up to a multiple of 4; y float32 [n][heads * dv]: the gated values before the norm; dtype: the model's.  single: every request
// brings one row; otherwise work buffers, C the rows of a chunk (kllm_ssd_chunk_rows) and chunk_bound an upper bound of the
// chunks: xc [n][channels rounded up to a multiple of 4] float32, or bfloat16 rounded up to a multiple of 8 with the
// tensor-core form; dt [chunk_bound][heads][C] float32, cum twice that; s_in [chunk_bound][heads][N][dv] float32; pairs
// [chunk_bound][groups][C][C] float32, or with the tensor-core form s_split [2][chunk_bound][heads][N][dv] bfloat16.
// early (single): the kernel may start beside the end of the one before it in the stream, which must write neither
// state nor ring.
extern "C" int kllm_ssd(float* y, const float* proj, int64_t stride, const float* conv_w, const float* conv_b,
                        const float* dt_bias, const float* a_log, const float* d, const int* q_start, const int* start_pos,
                        const int* state_slots, float* state, int64_t state_stride, float* ring, int64_t ring_stride, int n,
                        int n_requests, int heads, int groups, int N, int dv, int taps, int single, int early, int chunk_bound,
                        void* xc, float* dt, float* cum, float* pairs, float* s_in, void* s_split, int dtype, void* stream) {
    if (n <= 0 || n_requests <= 0) return 0;
    if (heads <= 0 || groups <= 0 || heads % groups || N <= 0 || dv <= 0) KLLM_FAIL("ssd: %d heads in %d groups of sizes %d, %d", heads, groups, N, dv);
    if (taps < 1 || taps > kC) KLLM_FAIL("ssd: a convolution of %d taps (up to %d)", taps, kC);
    if (heads > 65535 || groups > 65535 || n_requests > 65535) KLLM_FAIL("ssd: %d heads, %d requests in one launch", heads, n_requests);
    const bool tc = tensor_cores(dtype, N, dv);
    SsdArgs a;
    a.proj = proj; a.stride = stride; a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a_log = a_log; a.d = d;
    a.taps = taps; a.heads = heads; a.groups = groups; a.N = N; a.dv = dv; a.inner = heads * dv;
    a.channels = a.inner + 2 * groups * N; a.ch_pad = (a.channels + 3) / 4 * 4;
    a.q_start = q_start; a.start_pos = start_pos; a.state_slots = state_slots; a.n_requests = n_requests;
    a.state = state; a.state_stride = state_stride; a.ring = ring; a.ring_stride = ring_stride; a.y = y;
    a.xc = xc; a.xc_pad = tc ? (a.channels + 7) / 8 * 8 : a.ch_pad; a.dt = dt; a.cum = (float2*)cum; a.pairs = pairs; a.s_in = s_in;
    a.s_split = (bf16*)s_split; a.split_plane = (int64_t)chunk_bound * heads * N * dv;
    if (state_stride < (int64_t)heads * N * dv || ring_stride < (int64_t)taps * a.ch_pad)
        KLLM_FAIL("ssd: slots of %lld and %lld values are too small", (long long)state_stride, (long long)ring_stride);
    if (single && n != n_requests) KLLM_FAIL("ssd: %d rows of %d requests that bring one row each", n, n_requests);
    if (!single && (!xc || !dt || !cum || !s_in || chunk_bound <= 0 || !(tc ? s_split : (void*)pairs))) KLLM_FAIL("ssd: portions need work buffers");
    cudaStream_t s = (cudaStream_t)stream;
    const bool rows_vec = dv % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
    if (single) return rows_vec ? launch_step<4>(a, early != 0, s) : launch_step<1>(a, early != 0, s);
    a.vec = rows_vec && N % 4 == 0 && stride % 4 == 0 &&
            !(((uintptr_t)proj | (uintptr_t)xc | (uintptr_t)s_in | (uintptr_t)pairs | (uintptr_t)s_split | (uintptr_t)y) & 15);
    if (tc && !a.vec) KLLM_FAIL("ssd: the tensor-core form needs 16-byte aligned operands with row strides in multiples of 4");
    return tc ? run_portions_tc(a, chunk_bound, s) : run_portions(a, chunk_bound, s);
}

// out [n] rows of parts * w values in `dtype` at out_stride = y / rms(y) * gain, each of the `parts` pieces of a row by its own
// root mean square; y float32 [n][parts * w], gain float32 [parts * w].
extern "C" int kllm_part_norm(void* out, int64_t out_stride, const float* y, const float* gain, int n, int parts, int w, float eps,
                              int dtype, void* stream) {
    if (n <= 0) return 0;
    if (parts <= 0 || w <= 0) KLLM_FAIL("part norm: %d parts of %d values", parts, w);
    if ((int64_t)n * parts > 0x7fffffffLL) KLLM_FAIL("part norm: %d rows of %d parts in one launch", n, parts);
    // the form follows from the part's width and the addresses alone
    const bool warp = w <= 32 * 4 * kVec;
    const int threads = warp ? kThreads : (w <= 4096 ? 128 : kThreads), per_part = warp ? 32 : threads;
    const int esize = dtype == KLLM_F32 ? 4 : 2;
    const bool vec = w % 4 == 0 && w <= per_part * 4 * kVec && out_stride % 4 == 0 && !(((uintptr_t)y | (uintptr_t)gain) & 15) &&
                     !((uintptr_t)out & (4 * esize - 1));
    const int64_t items = (int64_t)n * parts;
    const int grid = (int)(warp ? (items + kThreads / 32 - 1) / (kThreads / 32) : items);
    cudaStream_t s = (cudaStream_t)stream;
#define KLLM_PN(T, VEC, WARP) \
    kllm_launch((part_norm_kernel<T, VEC, WARP>), dim3(grid), dim3(threads), 0, s, (T*)out, out_stride, y, gain, parts, w, eps, items)
#define KLLM_PN_T(T)                                       \
    if (warp && vec) KLLM_PN(T, true, true);               \
    else if (warp) KLLM_PN(T, false, true);                \
    else if (vec) KLLM_PN(T, true, false);                 \
    else KLLM_PN(T, false, false)
    if (dtype == KLLM_F32) {
        KLLM_PN_T(float);
    } else if (dtype == KLLM_BF16) {
        KLLM_PN_T(bf16);
    } else {
        KLLM_FAIL("part norm: unknown element type %d", dtype);
    }
#undef KLLM_PN_T
#undef KLLM_PN
    KLLM_LAUNCH_STATUS();
}
