// Linear attention with a decaying state, for mixed batches of prompt portions and single tokens, with
// the state of every request in a slot of a state tensor.
//
// Per head, with dk key channels d, dv value channels e and a state S [dk][dv] that starts at zero for
// a new request:
//
//     S_t[d][e] = alpha_t[d] S_(t-1)[d][e] + k_t[d] v_t[e]          o_t[e] = sum_d S_t[d][e] q_t[d]
//     y_t       = o_t / rms(o_t over the head's dv values) * gain * silu(g_t)
//
// The decay alpha has two forms.  Gated: alpha = sigmoid(z)^(1 / tau) per key channel, z = W2 low_t + b, the
// outer half of a low-rank product whose inner half `low` comes with the projections.  Fixed: one number per
// head.  q and k may be rotated first (the pairs (i, i + rot / 2), i < rot / 2, by position * freq[i], the angle
// formed in double precision) and are multiplied by q_scale and k_scale.  Everything is float32: the
// projections arrive unrounded, the decay, the state and every sum; y alone is stored in the model's type.
//
// Steps in which every request brings one row take one kernel (step_kernel): a cluster of CTAs per (head,
// request), each CTA with a slice of the value channels; the state's slice is on its way from HBM before the
// projections are waited for, is updated in registers and written back, and the cluster's CTAs join their sums
// of squares through distributed shared memory for the head's norm.
//
// Steps with portions take four kernels.  A request's rows are cut into chunks of kC rows.  With the cumulative decay
// D_ij = alpha_(j+1) ... alpha_i per key channel (D_ii = 1) and A_i = alpha_first ... alpha_i inside a chunk,
//
//     o_i   = sum_d (q_i A_i)[d] S_in[d] + sum over j <= i of W_ij v_j        W_ij = sum_d q_i[d] D_ij[d] k_j[d]
//     S_out = A_last S_in + sum over j of (k_j D_last,j) v_j^T
//
//   chunk_kernel   every (chunk, head) at once: W, q_i A_i, k_j D_last,j and A_last.  A thread carries k_j times its
//                  running decay from row to row, so no quotient of decays is ever formed: every factor is a product of
//                  numbers in [0, 1], and a decay that reaches zero inside a chunk is harmless
//   outer_kernel   every chunk at once: the chunk's own addition to the state
//   carry_kernel   the states at the chunks' starts, element by element over a request's chunks in order;
//                  moves the slot on
//   apply_kernel   every chunk at once: o, the head's norm and the gate
// Where a prompt is cut changes the order of float32 sums and nothing else.
#include "common.cuh"

KLLM_EXPORT_LAST_ERROR(gla)

namespace {

constexpr int kC = 64;          // rows of a chunk
constexpr int kThreads = 256;
constexpr int kMaxRot = 256;

struct GlaArgs {
    const float *q, *k, *v, *g;             // rows of the projections, float32, at `stride`
    int64_t stride;
    const float* low;                       // gated decay: [n][R] at `stride`; null: fixed decay
    const void* w2;                         // [H * dk][R] in the model's type
    const float* w2_bias;                   // [H * dk]
    int R;
    float inv_tau;
    const float* decay;                     // fixed decay: [H]
    const double* freq;                     // [rot / 2], or null
    int rot;
    float amplitude, q_scale, k_scale;
    const int* positions;
    const int *q_start, *state_slots;
    int n_requests, heads, dk, dv;
    float* state;
    int64_t state_stride;
    const float* gain;                      // [H * dv]
    float eps;
    void* y;
    int64_t y_stride;
    // work of the form for portions
    float *o, *qa, *kd, *a_last, *w, *s_in; // [n][H dv], [n][H dk] twice, [chunks][H dk], [chunks][H][kC][kC], [chunks][H][dk][dv]
    bool vec;                               // sizes and addresses allow 16-byte accesses throughout
    bool vec_out;                           // ... and four values of g, gain and y at once
    const int* start_pos;
};

__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}

__device__ __forceinline__ float peer_f32(const float* p, int rank) {
    unsigned a = (unsigned)__cvta_generic_to_shared(p), r;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(r) : "r"(a), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];\n" : "=f"(v) : "r"(r) : "memory");
    return v;
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
__device__ __forceinline__ float gated_alpha(float z, float inv_tau) {
    return expf(-(log1pf(expf(-fabsf(z))) + fmaxf(-z, 0.f)) * inv_tau);
}

// cos and sin of position * f in float32: the angle and its rest from whole turns in double precision
__device__ __forceinline__ void turn(int position, double f, float& c, float& s) {
    const double ang = (double)position * f;
    sincosf((float)(ang - rint(ang * 0.15915494309189533577) * 6.28318530717958647693), &s, &c);
}

// element d of a head's row, turned by the row's angles (cos [half], sin [half])
__device__ __forceinline__ float turned(const float* row, int d, int rot, const float* cs) {
    const float x = row[d];
    if (d >= rot) return x;
    const int half = rot >> 1;
    return d < half ? x * cs[d] - row[d + half] * cs[half + d] : x * cs[d - half] + row[d - half] * cs[d];
}

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
// grid (slices, heads, requests), cluster (slices, 1, 1).  Thread (cg, dl): V value channels e0 + cg V ..., key
// channels dl, dl + lanes, ...  Shared memory: partial sums [kThreads * V], o [sl], q, k, alpha [dk] each,
// cos / sin [rot], W2 [dk][R + 1] (gated).  Started early, the kernel reads the state before the kernel in front of it
// has ended: that kernel must not write the state.
template <typename T, int V>
__global__ void __launch_bounds__(kThreads)
step_kernel(const GlaArgs a, int sl) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    __shared__ float part;
    constexpr int NB = V == 4 ? 8 : 16;                     // key channels in flight per thread
    const int tid = threadIdx.x, slice = blockIdx.x, head = blockIdx.y, req = blockIdx.z;
    const int dk = a.dk, dv = a.dv, R = a.R;
    float* ps = sm;                                         // [kThreads * V], 16-byte aligned
    float* ob = ps + kThreads * V;                          // [sl]
    float* qs = ob + sl;
    float* ks = qs + dk;
    float* as = ks + dk;
    float* cs = as + dk;                                    // [rot]
    float* w2s = cs + a.rot;                                // [dk][R + 1]
    const int t = a.q_start[req];
    const int groups = sl / V, lanes = kThreads / groups, cg = tid % groups, dl = tid / groups;
    const bool on = dl < lanes;
    const int e = slice * sl + cg * V;
    float* Sg = a.state + (int64_t)a.state_slots[req] * a.state_stride + (int64_t)head * dk * dv + e;
    // what no kernel right before this one writes: the state, the decay's matrix, the angles
    Vec<V> s[NB];
#pragma unroll
    for (int i = 0; i < NB; i++) {
        const int d = dl + i * lanes;
        if (on && d < dk) s[i] = load_vec<V>(Sg + (int64_t)d * dv);
    }
    if (a.low) {
        const T* w2 = reinterpret_cast<const T*>(a.w2) + (int64_t)head * dk * R;
        for (int i = tid; i < dk * R; i += kThreads) w2s[(i / R) * (R + 1) + i % R] = to_f32(w2[i]);
    }
    const int half = a.rot >> 1;
    for (int i = tid; i < half; i += kThreads) {
        float c, sn;
        turn(a.positions[t], a.freq[i], c, sn);
        cs[i] = c * a.amplitude;
        cs[half + i] = sn * a.amplitude;
    }
    __syncthreads();
    griddep_wait();
    griddep_launch();
    const float* qr = a.q + (int64_t)t * a.stride + head * dk;
    const float* kr = a.k + (int64_t)t * a.stride + head * dk;
    for (int d = tid; d < dk; d += kThreads) {
        qs[d] = turned(qr, d, a.rot, cs) * a.q_scale;
        ks[d] = turned(kr, d, a.rot, cs) * a.k_scale;
        float al;
        if (a.low) {
            const float* lr = a.low + (int64_t)t * a.stride;
            float z = 0.f;
#pragma unroll 8
            for (int r = 0; r < R; r++) z = fmaf(lr[r], w2s[d * (R + 1) + r], z);
            al = gated_alpha(z + a.w2_bias[head * dk + d], a.inv_tau);
        } else {
            al = a.decay[head];
        }
        as[d] = al;
    }
    Vec<V> vv, acc;
#pragma unroll
    for (int j = 0; j < V; j++) acc.x[j] = 0.f;
    if (on) vv = load_vec<V>(a.v + (int64_t)t * a.stride + head * dv + e);
    __syncthreads();
    if (on) {
        for (int d0 = dl; d0 < dk; d0 += NB * lanes) {
            if (d0 != dl) {
#pragma unroll
                for (int i = 0; i < NB; i++) {
                    const int d = d0 + i * lanes;
                    if (d < dk) s[i] = load_vec<V>(Sg + (int64_t)d * dv);
                }
            }
#pragma unroll
            for (int i = 0; i < NB; i++) {
                const int d = d0 + i * lanes;
                if (d < dk) {
                    const float al = as[d], kd = ks[d], qd = qs[d];
#pragma unroll
                    for (int j = 0; j < V; j++) {
                        s[i].x[j] = fmaf(al, s[i].x[j], kd * vv.x[j]);
                        acc.x[j] = fmaf(qd, s[i].x[j], acc.x[j]);
                    }
                    store_vec<V>(Sg + (int64_t)d * dv, s[i]);
                }
            }
        }
        store_vec<V>(ps + dl * sl + cg * V, acc);
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < sl; c += kThreads) {
        float o = 0.f;
        for (int l = 0; l < lanes; l++) o += ps[l * sl + c];
        ob[c] = o;
        ss += o * o;
    }
    ss = block_sum(ss, red);
    if (tid == 0) part = ss;
    cluster_sync_all();
    float tot = 0.f;
    for (int r = 0; r < (int)gridDim.x; r++) tot += peer_f32(&part, r);
    const float scale = rsqrtf(tot / (float)dv + a.eps);
    T* yr = reinterpret_cast<T*>(a.y) + (int64_t)t * a.y_stride + head * dv + slice * sl;
    const float* gr = a.g + (int64_t)t * a.stride + head * dv + slice * sl;
    const float* gn = a.gain + head * dv + slice * sl;
    for (int c = tid; c < sl; c += kThreads) yr[c] = from_f32<T>(ob[c] * scale * gn[c] * silu_f(gr[c]));
    cluster_sync_all();                                     // no CTA leaves while another may still read its sum
}

// ---- portions ------------------------------------------------------------------------------------------------

// The request and first row of the step's chunk number `chunk`; false beyond the last chunk.
__device__ __forceinline__ bool find_chunk(const GlaArgs& a, int chunk, int& req, int& row0, int& rows, int& index) {
    for (req = 0; req < a.n_requests; req++) {
        const int lo = a.q_start[req], len = a.q_start[req + 1] - lo, chunks = (len + kC - 1) / kC;
        if (chunk < chunks) {
            index = chunk;
            row0 = lo + chunk * kC;
            rows = min(kC, len - chunk * kC);
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

// grid (chunk bound, heads).  Thread (j, g): row j of the chunk as a key, key channels (i * 4 + g) * 4 + 0 .. 3,
// i < DPT / 4.  Shared memory: k, then alpha [kC][4 DPT]; q [kC][4 DPT]; gated: W2 [dk][R + 1], low [kC][R].
template <typename T, int DPT, bool GATED>
__global__ void __launch_bounds__(kThreads)
chunk_kernel(const GlaArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int P = 4 * DPT;
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, j = tid >> 2, g = tid & 3, warp = tid >> 5;
    const int head = blockIdx.y, dk = a.dk, R = a.R, rot = a.rot, half = rot >> 1;
    int req, row0, rows, index;
    if (!find_chunk(a, blockIdx.x, req, row0, rows, index)) return;
    float* xs = sm;
    float* qs = xs + kC * P;
    float* w2s = qs + kC * P;
    float* lows = w2s + (GATED ? dk * (R + 1) : 0);
    const float* qg = a.q + (int64_t)row0 * a.stride + head * dk;
    const float* kg = a.k + (int64_t)row0 * a.stride + head * dk;
    if (a.vec) {
        for (int i = tid; i < kC * (P / 4); i += kThreads) {
            const int r = i / (P / 4), d = (i - r * (P / 4)) * 4;
            const bool in = r < rows && d < dk;
            const int64_t off = in ? r * a.stride + d : 0;
            cp_async16(qs + i * 4, qg + off, in);
            cp_async16(xs + i * 4, kg + off, in);
        }
    } else {
        for (int i = tid; i < kC * P; i += kThreads) {
            const int r = i / P, d = i - r * P;
            const bool in = r < rows && d < dk;
            qs[i] = in ? qg[r * a.stride + d] : 0.f;
            xs[i] = in ? kg[r * a.stride + d] : 0.f;
        }
    }
    cp_async_commit();
    if (GATED) {
        const T* w2 = reinterpret_cast<const T*>(a.w2) + (int64_t)head * dk * R;
        for (int i = tid; i < dk * R; i += kThreads) w2s[(i / R) * (R + 1) + i % R] = to_f32(w2[i]);
        for (int i = tid; i < rows * R; i += kThreads) lows[i] = a.low[(int64_t)(row0 + i / R) * a.stride + i % R];
    }
    cp_async_wait<0>();
    __syncthreads();
    if (half) {
        for (int i = tid; i < rows * half; i += kThreads) {
            const int r = i / half, d = i - r * half;
            float c, sn;
            turn(a.positions[row0 + r], a.freq[d], c, sn);
            c *= a.amplitude;
            sn *= a.amplitude;
            for (float* row : {qs + r * P, xs + r * P}) {
                const float u = row[d], v = row[d + half];
                row[d] = u * c - v * sn;
                row[d + half] = v * c + u * sn;
            }
        }
        __syncthreads();
    }
    float w[DPT];
#pragma unroll
    for (int i = 0; i < DPT; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(xs + j * P + (i + g) * 4);
        w[i] = k4.x * a.k_scale; w[i + 1] = k4.y * a.k_scale; w[i + 2] = k4.z * a.k_scale; w[i + 3] = k4.w * a.k_scale;
    }
    const float fixed = GATED ? 1.f : a.decay[head];
    if (GATED) {
        __syncthreads();                    // everyone has its keys: their place takes the decays
        for (int i = tid; i < rows * P; i += kThreads) {
            const int r = i / P, d = i - r * P;
            float al = 1.f;
            if (d < dk) {
                float z = 0.f;
#pragma unroll 4
                for (int u = 0; u < R; u++) z = fmaf(lows[r * R + u], w2s[d * (R + 1) + u], z);
                al = gated_alpha(z + a.w2_bias[head * dk + d], a.inv_tau);
            }
            xs[i] = al;
        }
        __syncthreads();
    }
    const int A_w = a.heads * dk;
    // q_i A_i and A_last, by the half of the threads whose keys have the fewer rows behind them
    if (tid >= kThreads / 2) {
        for (int d = tid - kThreads / 2; d < dk; d += kThreads / 2) {
            float c = 1.f;
            float* dst = a.qa + (int64_t)row0 * A_w + head * dk + d;
#pragma unroll 4
            for (int r = 0; r < rows; r++) {
                c *= GATED ? xs[r * P + d] : fixed;
                dst[(int64_t)r * A_w] = qs[r * P + d] * a.q_scale * c;
            }
            a.a_last[(int64_t)blockIdx.x * A_w + head * dk + d] = c;
        }
    }
    float* Wr = a.w + ((int64_t)blockIdx.x * a.heads + head) * kC * kC + j;
    const int jmin = warp * 8, jmax = jmin + 7;
    if (g == 0)
        for (int i = 0; i < min(jmin, rows); i++) Wr[i * kC] = 0.f;
    for (int i = jmin; i < rows; i++) {
        float acc = 0.f, acc2 = 0.f;
        const bool on = i > j;
#pragma unroll
        for (int u = 0; u < DPT; u += 4) {
            const float4 q4 = *reinterpret_cast<const float4*>(qs + i * P + (u + g) * 4);
            float4 al = make_float4(fixed, fixed, fixed, fixed);
            if (GATED) al = *reinterpret_cast<const float4*>(xs + i * P + (u + g) * 4);
            if (i > jmax) {                 // the same for the whole warp
                w[u] *= al.x; w[u + 1] *= al.y; w[u + 2] *= al.z; w[u + 3] *= al.w;
            } else if (on) {
                w[u] *= al.x; w[u + 1] *= al.y; w[u + 2] *= al.z; w[u + 3] *= al.w;
            }
            acc = fmaf(q4.x, w[u], acc);
            acc2 = fmaf(q4.y, w[u + 1], acc2);
            acc = fmaf(q4.z, w[u + 2], acc);
            acc2 = fmaf(q4.w, w[u + 3], acc2);
        }
        acc += acc2;
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        if (g == 0) Wr[i * kC] = i >= j ? acc * a.q_scale : 0.f;
    }
    if (j < rows) {
        float* dst = a.kd + (int64_t)(row0 + j) * A_w + head * dk;
#pragma unroll
        for (int i = 0; i < DPT; i += 4) {
            const int d = (i + g) * 4;
            if (a.vec) {
                if (d < dk) *reinterpret_cast<float4*>(dst + d) = make_float4(w[i], w[i + 1], w[i + 2], w[i + 3]);
            } else {
#pragma unroll
                for (int u = 0; u < 4; u++)
                    if (d + u < dk) dst[d + u] = w[i + u];
            }
        }
    }
}

// N consecutive values of shared memory as the register tile of thread `t` of 16: fours at 64 u + 4 t (N 4, 8), or two at 2 t
template <int N> __device__ __forceinline__ int tile_at(int t, int i) { return N == 2 ? 2 * t + i : (i >> 2) * 64 + 4 * t + (i & 3); }

// grid (chunk bound, heads, tiles of 16 RM key channels by 16 RN value channels): s_in = sum over the chunk's rows of
// kd_j v_j^T.  Thread (ty, tx): an RM x RN tile.  Shared memory: kd [kC][16 RM], v [kC][16 RN].
template <int RM, int RN>
__global__ void __launch_bounds__(kThreads)
outer_kernel(const GlaArgs a, int e_tiles) {
    extern __shared__ __align__(16) float sm[];
    constexpr int TM = 16 * RM, TN = 16 * RN;
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int head = blockIdx.y, d0 = blockIdx.z / e_tiles * TM, e0 = blockIdx.z % e_tiles * TN, dk = a.dk, dv = a.dv;
    int req, row0, rows, index;
    if (!find_chunk(a, blockIdx.x, req, row0, rows, index)) return;
    float* ks = sm;
    float* vs = ks + kC * TM;
    const int A_w = a.heads * dk;
    const float* kg = a.kd + (int64_t)row0 * A_w + head * dk + d0;
    const float* vg = a.v + (int64_t)row0 * a.stride + head * dv + e0;
    if (a.vec) {
        for (int i = tid; i < rows * (TM / 4); i += kThreads) {
            const int r = i / (TM / 4), d = (i - r * (TM / 4)) * 4;
            cp_async16(ks + r * TM + d, kg + (d0 + d < dk ? (int64_t)r * A_w + d : 0), d0 + d < dk);
        }
        for (int i = tid; i < rows * (TN / 4); i += kThreads) {
            const int r = i / (TN / 4), c = (i - r * (TN / 4)) * 4;
            cp_async16(vs + r * TN + c, vg + (e0 + c < dv ? (int64_t)r * a.stride + c : 0), e0 + c < dv);
        }
        cp_async_commit();
        cp_async_wait<0>();
    } else {
        for (int i = tid; i < rows * TM; i += kThreads) {
            const int r = i / TM, d = i - r * TM;
            ks[i] = d0 + d < dk ? kg[(int64_t)r * A_w + d] : 0.f;
        }
        for (int i = tid; i < rows * TN; i += kThreads) {
            const int r = i / TN, c = i - r * TN;
            vs[i] = e0 + c < dv ? vg[(int64_t)r * a.stride + c] : 0.f;
        }
    }
    __syncthreads();
    float acc[RM][RN];
#pragma unroll
    for (int m = 0; m < RM; m++)
#pragma unroll
        for (int n = 0; n < RN; n++) acc[m][n] = 0.f;
#pragma unroll 2
    for (int r = 0; r < rows; r++) {
        float k[RM], v[RN];
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
            v[4 * u] = t.x; v[4 * u + 1] = t.y; v[4 * u + 2] = t.z; v[4 * u + 3] = t.w;
        }
#pragma unroll
        for (int m = 0; m < RM; m++)
#pragma unroll
            for (int n = 0; n < RN; n++) acc[m][n] = fmaf(k[m], v[n], acc[m][n]);
    }
    float* S = a.s_in + ((int64_t)blockIdx.x * a.heads + head) * dk * dv;
#pragma unroll
    for (int m = 0; m < RM; m++) {
        const int d = d0 + tile_at<RM>(ty, m);
        if (d >= dk) continue;
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
// states at their starts.
template <int V>
__global__ void __launch_bounds__(kThreads)
carry_kernel(const GlaArgs a) {
    griddep_wait();
    griddep_launch();
    const int head = blockIdx.y, req = blockIdx.z, dk = a.dk, dv = a.dv;
    const int64_t i = ((int64_t)blockIdx.x * kThreads + threadIdx.x) * V;
    if (i >= (int64_t)dk * dv) return;
    int chunk = 0;
    for (int r = 0; r < req; r++) chunk += (a.q_start[r + 1] - a.q_start[r] + kC - 1) / kC;
    const int chunks = (a.q_start[req + 1] - a.q_start[req] + kC - 1) / kC;
    float* slot = a.state + (int64_t)a.state_slots[req] * a.state_stride + (int64_t)head * dk * dv + i;
    float* w = a.s_in + ((int64_t)chunk * a.heads + head) * dk * dv + i;
    const float* al = a.a_last + (int64_t)chunk * a.heads * dk + head * dk + i / dv;
    const int64_t step = (int64_t)a.heads * dk * dv;
    const int a_step = a.heads * dk;
    Vec<V> s = load_vec<V>(slot);
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        Vec<V> loc[AHEAD];
        float d[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                loc[u] = load_vec<V>(w + (c0 + u) * step);
                d[u] = al[(int64_t)(c0 + u) * a_step];
            }
#pragma unroll
        for (int u = 0; u < AHEAD; u++)
            if (c0 + u < chunks) {
                store_vec<V>(w + (c0 + u) * step, s);
#pragma unroll
                for (int j = 0; j < V; j++) s.x[j] = fmaf(d[u], s.x[j], loc[u].x[j]);
            }
    }
    store_vec<V>(slot, s);
}

// grid (chunk bound, heads, column blocks of 64 NJ): o = [q A | W] [S_in ; v], in blocks of kKB inner elements, two of them
// in shared memory.  Thread (rg, cg): rows 4 rg .. 4 rg + 3, value channels j * 64 + 4 cg .. + 3.  NORM: the columns are all
// of the head's (grid.z is 1) and the row is normed, gated and stored in y; otherwise o is stored.
// Shared memory, twice: left [kC][kKB + 4], right [kKB][64 NJ].
constexpr int kKB = 32;

template <typename T, int NJ, bool NORM>
__global__ void __launch_bounds__(kThreads)
apply_kernel(const GlaArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int QP = kKB + 4, CW = 64 * NJ, STAGE = kC * QP + kKB * CW;
    griddep_wait();
    griddep_launch();
    const int tid = threadIdx.x, cg = tid & 15, rg = tid >> 4;
    const int head = blockIdx.y, e0 = blockIdx.z * CW, dk = a.dk, dv = a.dv;
    const int ne = min(CW, dv - e0);
    int req, row0, rows, index;
    if (!find_chunk(a, blockIdx.x, req, row0, rows, index)) return;
    float acc[4][NJ * 4];
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int j = 0; j < NJ * 4; j++) acc[r][j] = 0.f;
    const int A_w = a.heads * dk, B_w = a.heads * dv;
    const bool from_zero = index == 0 && a.start_pos[req] == 0;        // the state in front of a request's first chunk
    const int nb_s = from_zero ? 0 : (dk + kKB - 1) / kKB, nb = nb_s + (rows + kKB - 1) / kKB;
    const float* S = a.s_in + ((int64_t)blockIdx.x * a.heads + head) * dk * dv + e0;
    const float* W = a.w + ((int64_t)blockIdx.x * a.heads + head) * kC * kC;
    auto load = [&](int b) {                // inner elements k0 .. k0 + kKB - 1 of the state's part, then of the chunk's own
        float* left = sm + (b & 1) * STAGE;
        float* right = left + kC * QP;
        const bool state = b < nb_s;
        const int k0 = (state ? b : b - nb_s) * kKB, nk = min(kKB, (state ? dk : rows) - k0);
        const float* lg = state ? a.qa + (int64_t)row0 * A_w + head * dk + k0 : W + k0;
        const float* rg_ = state ? S + (int64_t)k0 * dv : a.v + (int64_t)(row0 + k0) * a.stride + head * dv + e0;
        const int64_t ls = state ? A_w : kC, rs = state ? dv : a.stride;
        if (a.vec) {
            for (int i = tid; i < kC * (kKB / 4); i += kThreads) {
                const int r = i / (kKB / 4), k = (i - r * (kKB / 4)) * 4;
                const bool in = r < rows && (state ? k < nk : true);      // W's rows are whole: zeros beyond the diagonal
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
        const float* qs = sm + (b & 1) * STAGE;
        const float* ss = qs + kC * QP;
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
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int row = rg * 4 + r;
        float sq = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; j++)
#pragma unroll
            for (int c = 0; c < 4; c++) {
                const int col = j * 64 + cg * 4 + c;
                if (col >= ne) acc[r][j * 4 + c] = 0.f;
                sq += acc[r][j * 4 + c] * acc[r][j * 4 + c];
            }
        if constexpr (NORM) {
#pragma unroll
            for (int o = 8; o >= 1; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
            if (row < rows) {
                const float scale = rsqrtf(sq / (float)dv + a.eps);
                T* yr = reinterpret_cast<T*>(a.y) + (int64_t)(row0 + row) * a.y_stride + head * dv;
                const float* gr = a.g + (int64_t)(row0 + row) * a.stride + head * dv;
                const float* gn = a.gain + head * dv;
#pragma unroll
                for (int j = 0; j < NJ; j++) {
                    const int col = j * 64 + cg * 4;
                    float v[4] = {acc[r][j * 4] * scale, acc[r][j * 4 + 1] * scale, acc[r][j * 4 + 2] * scale, acc[r][j * 4 + 3] * scale};
                    if (a.vec_out) {
                        if (col >= ne) continue;
                        const float4 g4 = *reinterpret_cast<const float4*>(gr + col), n4 = *reinterpret_cast<const float4*>(gn + col);
                        v[0] *= n4.x * silu_f(g4.x); v[1] *= n4.y * silu_f(g4.y);
                        v[2] *= n4.z * silu_f(g4.z); v[3] *= n4.w * silu_f(g4.w);
                        if constexpr (sizeof(T) == 4) {
                            *reinterpret_cast<float4*>(yr + col) = make_float4(v[0], v[1], v[2], v[3]);
                        } else {
                            __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
                            uint2 pk;
                            pk.x = *reinterpret_cast<uint32_t*>(&lo);
                            pk.y = *reinterpret_cast<uint32_t*>(&hi);
                            *reinterpret_cast<uint2*>(yr + col) = pk;
                        }
                    } else {
#pragma unroll
                        for (int c = 0; c < 4; c++)
                            if (col + c < ne) yr[col + c] = from_f32<T>(v[c] * gn[col + c] * silu_f(gr[col + c]));
                    }
                }
            }
        } else if (row < rows) {
            float* orow = a.o + (int64_t)(row0 + row) * B_w + head * dv + e0;
#pragma unroll
            for (int j = 0; j < NJ; j++)
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const int col = j * 64 + cg * 4 + c;
                    if (col < ne) orow[col] = acc[r][j * 4 + c];
                }
        }
    }
}

// a head wider than one apply CTA: norm and gate in a kernel of their own, one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(kThreads)
norm_gate_kernel(const GlaArgs a, int n) {
    griddep_wait();
    griddep_launch();
    const int lane = threadIdx.x & 31, dv = a.dv;
    const int64_t item = (int64_t)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
    if (item >= (int64_t)n * a.heads) return;
    const int64_t t = item / a.heads;
    const int head = (int)(item - t * a.heads);
    const float* orow = a.o + item * dv;
    float sq = 0.f;
    for (int c = lane; c < dv; c += 32) sq += orow[c] * orow[c];
    const float scale = rsqrtf(warp_sum(sq) / (float)dv + a.eps);
    const float* gr = a.g + t * a.stride + head * dv;
    T* yr = reinterpret_cast<T*>(a.y) + t * a.y_stride + head * dv;
    for (int c = lane; c < dv; c += 32) yr[c] = from_f32<T>(orow[c] * scale * a.gain[head * dv + c] * silu_f(gr[c]));
}

template <int V> size_t step_smem(const GlaArgs& a, int sl) {
    return sizeof(float) * ((size_t)3 * a.dk + a.rot + sl + (size_t)kThreads * V + (a.low ? (size_t)a.dk * (a.R + 1) : 0));
}

template <typename T, int V>
int launch_step(const GlaArgs& a, bool early, cudaStream_t s) {
    // slices: a power of two up to a portable cluster's 8 CTAs, more of them while the launch would leave SMs idle
    int slices = 1;
    auto splits = [&](int n) { return a.dv % (n * V) == 0; };
    while (a.dv / slices / V > kThreads && slices < 8 && splits(slices * 2)) slices *= 2;
    while (slices < 8 && splits(slices * 2) && a.dv / (slices * 2) >= 16 && (int64_t)slices * a.heads * a.n_requests < 148) slices *= 2;
    const int sl = a.dv / slices;
    if (sl / V > kThreads) KLLM_FAIL("gla step: a head of %d value channels does not fit", a.dv);
    const size_t smem = step_smem<V>(a, sl);
    if (smem > 200 * 1024) KLLM_FAIL("gla step: a head of %d key channels with a decay of rank %d does not fit shared memory", a.dk, a.R);
    auto kern = step_kernel<T, V>;
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) KLLM_FAIL("gla step: %s", cudaGetErrorString(e));
        raised = true;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(slices, a.heads, a.n_requests);
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = slices;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = (early && kllm_pdl_enabled()) ? 2 : 1;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kern, a, sl);
    if (e != cudaSuccess) KLLM_FAIL("gla step: %s", cudaGetErrorString(e));
    KLLM_LAUNCH_STATUS();
}

template <typename K>
int raise_smem(K kern, bool& raised) {
    if (raised) return 0;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) KLLM_FAIL("gla: %s", cudaGetErrorString(e));
    raised = true;
    return 0;
}

template <typename T, int DPT, bool GATED>
int launch_chunk(const GlaArgs& a, int chunk_bound, cudaStream_t s) {
    const size_t smem = sizeof(float) * ((size_t)2 * kC * 4 * DPT +
                                         (GATED ? (size_t)kC * a.R + (size_t)a.dk * (a.R + 1) : 0));
    if (smem > 220 * 1024) KLLM_FAIL("gla: a head of %d key channels with a decay of rank %d does not fit shared memory", a.dk, a.R);
    static bool raised = false;
    int rc = raise_smem(chunk_kernel<T, DPT, GATED>, raised);
    if (rc) return rc;
    kllm_launch_dep(false, (chunk_kernel<T, DPT, GATED>), dim3(chunk_bound, a.heads), dim3(kThreads), smem, s, a);
    KLLM_LAUNCH_STATUS();
}

template <typename T, int DPT>
int launch_chunk(const GlaArgs& a, int chunk_bound, cudaStream_t s) {
    return a.low ? launch_chunk<T, DPT, true>(a, chunk_bound, s) : launch_chunk<T, DPT, false>(a, chunk_bound, s);
}

template <int RM, int RN>
int launch_outer(const GlaArgs& a, int chunk_bound, cudaStream_t s) {
    const int e_tiles = (a.dv + 16 * RN - 1) / (16 * RN), d_tiles = (a.dk + 16 * RM - 1) / (16 * RM);
    static bool raised = false;
    int rc = raise_smem(outer_kernel<RM, RN>, raised);
    if (rc) return rc;
    kllm_launch_dep(false, (outer_kernel<RM, RN>), dim3(chunk_bound, a.heads, e_tiles * d_tiles), dim3(kThreads),
                    sizeof(float) * kC * 16 * (RM + RN), s, a, e_tiles);
    KLLM_LAUNCH_STATUS();
}

template <typename T, int NJ, bool NORM>
int launch_apply(const GlaArgs& a, int chunk_bound, cudaStream_t s) {
    const size_t smem = sizeof(float) * 2 * (kC * (kKB + 4) + kKB * 64 * NJ);
    static bool raised = false;
    int rc = raise_smem(apply_kernel<T, NJ, NORM>, raised);
    if (rc) return rc;
    kllm_launch_dep(false, (apply_kernel<T, NJ, NORM>), dim3(chunk_bound, a.heads, NORM ? 1 : (a.dv + 64 * NJ - 1) / (64 * NJ)),
                    dim3(kThreads), smem, s, a);
    KLLM_LAUNCH_STATUS();
}

template <typename T>
int run(GlaArgs a, int n, bool single, bool early, int chunk_bound, cudaStream_t s) {
    const bool rows_vec = a.dv % 4 == 0 && a.stride % 4 == 0 && a.state_stride % 4 == 0 &&
                          !(((uintptr_t)a.state | (uintptr_t)a.v) & 15);
    if (single) return rows_vec ? launch_step<T, 4>(a, early, s) : launch_step<T, 1>(a, early, s);
    a.vec = rows_vec && a.dk % 4 == 0 && !(((uintptr_t)a.s_in | (uintptr_t)a.qa | (uintptr_t)a.kd | (uintptr_t)a.w | (uintptr_t)a.q | (uintptr_t)a.k) & 15);
    a.vec_out = a.vec && a.y_stride % 4 == 0 && !(((uintptr_t)a.g | (uintptr_t)a.gain | (uintptr_t)a.y) & 15);
    const bool vec = a.vec;
    int rc;
    if (a.dk <= 32) rc = launch_chunk<T, 8>(a, chunk_bound, s);
    else if (a.dk <= 64) rc = launch_chunk<T, 16>(a, chunk_bound, s);
    else if (a.dk <= 128) rc = launch_chunk<T, 32>(a, chunk_bound, s);
    else rc = launch_chunk<T, 64>(a, chunk_bound, s);
    if (rc) return rc;
    if (a.dk <= 32) rc = a.dv <= 64 ? launch_outer<2, 4>(a, chunk_bound, s) : launch_outer<2, 8>(a, chunk_bound, s);
    else if (a.dk <= 64) rc = a.dv <= 64 ? launch_outer<4, 4>(a, chunk_bound, s) : launch_outer<4, 8>(a, chunk_bound, s);
    else rc = a.dv <= 64 ? launch_outer<8, 4>(a, chunk_bound, s) : launch_outer<8, 8>(a, chunk_bound, s);
    if (rc) return rc;
    const int64_t elems = (int64_t)a.dk * a.dv;
    if (vec)
        kllm_launch_dep(false, (carry_kernel<4>), dim3((unsigned)((elems / 4 + kThreads - 1) / kThreads), a.heads, a.n_requests),
                        dim3(kThreads), 0, s, a);
    else
        kllm_launch_dep(false, (carry_kernel<1>), dim3((unsigned)((elems + kThreads - 1) / kThreads), a.heads, a.n_requests),
                        dim3(kThreads), 0, s, a);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) KLLM_FAIL("gla: %s", cudaGetErrorString(e));
    if (a.dv <= 64) return launch_apply<T, 1, true>(a, chunk_bound, s);
    if (a.dv <= 128) return launch_apply<T, 2, true>(a, chunk_bound, s);
    if (a.dv <= 256) return launch_apply<T, 4, true>(a, chunk_bound, s);
    rc = launch_apply<T, 4, false>(a, chunk_bound, s);
    if (rc) return rc;
    const int64_t items = (int64_t)n * a.heads;
    kllm_launch((norm_gate_kernel<T>), dim3((unsigned)((items + 7) / 8)), dim3(kThreads), 0, s, a, n);
    KLLM_LAUNCH_STATUS();
}

}  // namespace

extern "C" int kllm_gla_chunk_rows() { return kC; }

// q, k float32 rows of heads * dk, v, g rows of heads * dv, low rows of R values (null: the fixed decay), all at row
// stride `stride`; w2 [heads * dk][R] in the element type `dtype`, w2_bias float32 [heads * dk]; decay float32 [heads];
// freq double [rot / 2] or null; state float32 [slots][state_stride] whose first heads * dk * dv values are S as
// [heads][dk][dv]; gain float32 [heads * dv]; y in `dtype` at row stride y_stride.  single: every request brings one
// row; otherwise the work buffers qa, kd [n][heads dk], a_last [chunk_bound][heads dk], w [chunk_bound][heads][C][C] (C:
// rows of a chunk), s_in [chunk_bound][heads][dk][dv] and, for dv above 256, o [n][heads dv] are float32 and chunk_bound an upper bound of the chunks (sum over requests of
// ceil(rows / kllm_gla_chunk_rows())).  early (single): the kernel may start beside the end of the one before it in the
// stream, which must not write the state.
extern "C" int kllm_gla(void* y, int64_t y_stride, const float* q, const float* k, const float* v, const float* g, int64_t stride,
                        const float* low, const void* w2, const float* w2_bias, int R, float inv_tau, const float* decay,
                        const double* freq, int rot, float amplitude, float q_scale, float k_scale, const int* positions,
                        const int* q_start, const int* start_pos, const int* state_slots, float* state, int64_t state_stride,
                        const float* gain, float eps, int n, int n_requests, int heads, int dk, int dv, int single,
                        int early, int chunk_bound, float* o, float* qa, float* kd, float* a_last, float* w, float* s_in, int dtype, void* stream) {
    if (n <= 0 || n_requests <= 0) return 0;
    if (heads <= 0 || dk <= 0 || dk > 256 || dv <= 0) KLLM_FAIL("gla: %d heads of sizes %d (up to 256), %d", heads, dk, dv);
    if (heads > 65535 || n_requests > 65535) KLLM_FAIL("gla: %d heads, %d requests in one launch", heads, n_requests);
    if (rot < 0 || (rot & 1) || rot > dk || rot > kMaxRot || (rot > 0 && !freq)) KLLM_FAIL("gla: rotary width %d invalid for head size %d", rot, dk);
    if (low ? (!w2 || !w2_bias || R <= 0) : !decay) KLLM_FAIL("gla: a decay needs its matrix and bias, or one number per head");
    if (state_stride < (int64_t)heads * dk * dv) KLLM_FAIL("gla: a state slot of %lld values is too small", (long long)state_stride);
    if (single && n != n_requests) KLLM_FAIL("gla: %d rows of %d requests that bring one row each", n, n_requests);
    if (!single && (!qa || !kd || !a_last || !w || !s_in || (dv > 256 && !o) || chunk_bound <= 0)) KLLM_FAIL("gla: portions need work buffers");
    GlaArgs a;
    a.q = q; a.k = k; a.v = v; a.g = g; a.stride = stride; a.low = low; a.w2 = w2; a.w2_bias = w2_bias; a.R = low ? R : 0;
    a.inv_tau = inv_tau; a.decay = decay; a.freq = freq; a.rot = rot; a.amplitude = amplitude; a.q_scale = q_scale;
    a.k_scale = k_scale; a.positions = positions; a.q_start = q_start; a.state_slots = state_slots; a.n_requests = n_requests;
    a.heads = heads; a.dk = dk; a.dv = dv; a.state = state; a.state_stride = state_stride; a.gain = gain; a.eps = eps; a.y = y;
    a.y_stride = y_stride; a.o = o; a.qa = qa; a.kd = kd; a.a_last = a_last; a.w = w; a.s_in = s_in; a.vec = a.vec_out = false; a.start_pos = start_pos;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KLLM_F32) return run<float>(a, n, single != 0, early != 0, chunk_bound, s);
    if (dtype == KLLM_BF16) return run<bf16>(a, n, single != 0, early != 0, chunk_bound, s);
    KLLM_FAIL("gla: unknown element type %d", dtype);
}
