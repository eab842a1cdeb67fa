// Kernels of two recurrences whose gates depend on the token: the per-channel decays of gated linear attention (a low-rank map, a
// sigmoid, a root; the recurrence itself is channel_decay_scan_kernel), and a diagonal recurrence with a real gate per channel
// behind a short convolution (Griffin's RG-LRU).
// Included by hybrid_ops.cu inside namespace b200h, after its helpers and token_shift.cuh (softplus32).
//
// Number formats: projections (T) are read once; decays, gates, the recurrence and its state are float.  The convolution's output u
// is T: it is the operand of the gates' block-diagonal product, and the recurrence reads the same rounded values.

// V consecutive values of T as float / back
template <int V> __device__ __forceinline__ void load_vals(const float* p, float (&o)[V])
{
    if (V == 2) { const float2 v = *reinterpret_cast<const float2*>(p); o[0] = v.x; o[V - 1] = v.y; } else o[0] = p[0];
}
template <int V> __device__ __forceinline__ void load_vals(const bf16* p, float (&o)[V])
{
    if (V == 2) {
        const unsigned raw = *reinterpret_cast<const unsigned*>(p);
        o[0] = __uint_as_float(raw << 16);
        o[V - 1] = __uint_as_float(raw & 0xffff0000u);
    } else o[0] = to_f(p[0]);
}
template <int V> __device__ __forceinline__ void store_vals(float* p, const float (&v)[V])
{
    if (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[V - 1]); else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void store_vals(bf16* p, const float (&v)[V])
{
    if (V == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[V - 1]); else p[0] = from_f<bf16>(v[0]);
}

// z = sum_k a[k, c] low[t, k] + bias[c];  decay[t, c] = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau), or, with a rate per head of `dim`
// channels, exp(-rate[c / dim] softplus(z)).  A block takes ROWS rows and
// V * blockDim.x channels; the rows' low-rank vectors sit in shared memory as [rank][ROWS], a thread reads its V columns of `a` once
// for all of them and keeps ROWS * V sums in registers.
template <typename T, int ROWS, int V>
__global__ void __launch_bounds__(128) low_rank_decay_kernel(const T* __restrict__ low, int64_t ld, const T* __restrict__ a,
                                                            const float* __restrict__ bias, int n, int channels, int rank, float inv_tau,
                                                            const float* __restrict__ rate, int dim, float* __restrict__ decay)
{
    extern __shared__ __align__(16) float lrd_smem[];
    constexpr int Q = ROWS % 4 == 0 ? 4 : 1;                  // rows per shared-memory read
    const int t0 = blockIdx.y * ROWS, c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    for (int i = threadIdx.x; i < rank * ROWS; i += blockDim.x) {
        const int r = i / rank, k = i - r * rank;
        lrd_smem[k * ROWS + r] = t0 + r < n ? to_f(low[(size_t)(t0 + r) * ld + k]) : 0.f;
    }
    __syncthreads();
    if (c >= channels) return;
    float z[ROWS][V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
        const float b = bias[c + e];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) z[r][e] = b;
    }
#pragma unroll 8
    for (int k = 0; k < rank; ++k) {
        float w[V];
        load_vals<V>(a + (size_t)k * channels + c, w);
#pragma unroll
        for (int r = 0; r < ROWS; r += Q) {
            float v[Q];
            if (Q == 4) {
                const float4 q = *reinterpret_cast<const float4*>(lrd_smem + k * ROWS + r);
                v[0] = q.x; v[1 % Q] = q.y; v[2 % Q] = q.z; v[3 % Q] = q.w;
            } else {
                v[0] = lrd_smem[k * ROWS + r];
            }
#pragma unroll
            for (int q = 0; q < Q; ++q)
#pragma unroll
                for (int e = 0; e < V; ++e) z[r + q][e] = fmaf(w[e], v[q], z[r + q][e]);
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (t0 + r < n) {
            float d[V];
#pragma unroll
            for (int e = 0; e < V; ++e) d[e] = rate ? expf(-rate[(c + e) / dim] * softplus32(z[r][e])) : expf(-softplus32(-z[r][e]) * inv_tau);
            store_vals<V>(decay + (size_t)(t0 + r) * channels + c, d);
        }
    }
}

// 0.5 z (1 + tanh(w)) = z sigmoid(2 w), w = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_f(float z)
{
    return z / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));              // 2 sqrt(2 / pi)
}

// u[t, c] = conv_bias[c] + sum_j w[c, j] * v[t - taps + 1 + j, c] with v = x + x_bias; v before a sequence's rows of this step comes from
// its state (the last taps - 1 values, oldest first; zeros at a sequence's start because a fresh slot is zeroed).  A thread owns V
// channels and walks ROWS consecutive rows of the step with the last TAPS values in registers (TAPS >= taps: leading weights zero);
// the rows' loads are issued before any is used.  The state is advanced later, by the scan that follows.
template <typename T, int TAPS, int ROWS, int V>
__global__ void __launch_bounds__(128) gated_conv_kernel(const T* __restrict__ x, int64_t ld, const float* __restrict__ x_bias,
                                                        const float* __restrict__ w, const float* __restrict__ conv_bias, int taps,
                                                        const float* __restrict__ state, int64_t slot_stride, const int* __restrict__ tok_seq,
                                                        const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int n, int width,
                                                        T* __restrict__ u)
{
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V, t0 = blockIdx.y * ROWS;
    if (c >= width) return;
    const int rows = min(ROWS, n - t0);
    float xv[ROWS][V], wt[V][TAPS], win[TAPS][V], xb[V], cb[V];
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (r < rows) load_vals<V>(x + (size_t)(t0 + r) * ld + c, xv[r]);
#pragma unroll
    for (int e = 0; e < V; ++e) {
        xb[e] = x_bias ? x_bias[c + e] : 0.f;
        cb[e] = conv_bias ? conv_bias[c + e] : 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wt[e][j] = j >= TAPS - taps ? w[(size_t)(c + e) * taps + j - (TAPS - taps)] : 0.f;
    }
    int seq = -1;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (r < rows) {
            const int s = tok_seq[t0 + r];
            if (s != seq) {                                   // this block's first row of the sequence: the window from its earlier rows or its state
                seq = s;
                const int first = cu_q[s], local = t0 + r - first;
                const float* st = state + (int64_t)seq_slot[s] * slot_stride;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int src = local - (TAPS - 1) + j;
#pragma unroll
                    for (int e = 0; e < V; ++e) win[j][e] = 0.f;
                    if (j >= TAPS - taps) {
                        if (src >= 0) {
                            load_vals<V>(x + (size_t)(first + src) * ld + c, win[j]);
#pragma unroll
                            for (int e = 0; e < V; ++e) win[j][e] += xb[e];
                        } else {
#pragma unroll
                            for (int e = 0; e < V; ++e) win[j][e] = st[(size_t)(src + taps - 1) * width + c + e];
                        }
                    }
                }
            }
            float acc[V];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                win[TAPS - 1][e] = xv[r][e] + xb[e];
                acc[e] = cb[e];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(wt[e][j], win[j][e], acc[e]);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) win[j][e] = win[j + 1][e];
            }
            store_vals<V>(u + (size_t)(t0 + r) * width + c, acc);
        }
    }
}

struct GatedScan {
    const float* z;           // [blocks, n, 2 * bw]
    const float* r_bias;
    const float* i_bias;
    const float* lam;
    float* state;
    int64_t slot_stride;
    const int* cu_q;
    const int* seq_slot;
    int n, width, bw, taps;   // bw = width / blocks
    float rate;
    int64_t ld;
    const float* x_bias;
    const float* y_bias;
    float* conv_state;
};

// Per channel, with r, i the sigmoids of the two gates:  log a = -rate r softplus(lam),  S <- a S + sqrt(1 - a^2) i u,
// out = S gelu(y + y_bias).  The recurrence is linear in S, so a block scans time in parallel: thread (lane, w) owns channel
// blockIdx.x * blockDim.x + lane and rows [w R, w R + R) of a tile of blockDim.y * R rows; it folds its rows into one pair (product of
// the a's, state from zero), the pairs meet in shared memory (double-buffered: one barrier per tile), every thread folds those before
// its own into its incoming state and replays its rows from registers.  Every input is read once.  A launch for steps of single rows
// has blockDim.y = 1: no shared memory, no barrier.
// Afterwards the thread of row group 0 advances the convolution's state of its channel (it reads all it needs and then writes).
template <typename T, int R>
__global__ void __launch_bounds__(512) real_gated_scan_kernel(GatedScan g, const T* __restrict__ x, const T* __restrict__ y,
                                                             const T* __restrict__ u, T* __restrict__ out)
{
    extern __shared__ __align__(16) float rgs_smem[];
    const int lane = threadIdx.x, w = threadIdx.y, X = blockDim.x, NW = blockDim.y;
    const int s = blockIdx.y, first = g.cu_q[s], last = g.cu_q[s + 1];
    if (first == last) return;                                // the whole block leaves
    const int c_raw = blockIdx.x * X + lane;
    const bool live = c_raw < g.width;
    const int c = live ? c_raw : g.width - 1;
    const float rb = g.r_bias ? g.r_bias[c] : 0.f, ib = g.i_bias ? g.i_bias[c] : 0.f, yb = g.y_bias ? g.y_bias[c] : 0.f;
    const float slope = -g.rate * softplus32(g.lam[c]);
    const int b = c / g.bw;
    const float* zr = g.z + (size_t)b * g.n * 2 * g.bw + (c - b * g.bw);
    float* sp = g.state + (int64_t)g.seq_slot[s] * g.slot_stride;
    float carry = sp[c];
    int p = 0;
    for (int t0 = first; t0 < last; t0 += NW * R, p ^= 1) {
        const int tb = t0 + w * R;
        float a[R], v[R], yv[R];
#pragma unroll
        for (int k = 0; k < R; ++k) {
            a[k] = v[k] = yv[k] = 0.f;
            if (tb + k < last) {
                const size_t t = (size_t)(tb + k);
                a[k] = zr[t * 2 * g.bw];
                v[k] = zr[t * 2 * g.bw + g.bw];
                yv[k] = to_f(y[t * g.ld + c]);
            }
        }
        float uv[R];
#pragma unroll
        for (int k = 0; k < R; ++k) uv[k] = tb + k < last ? to_f(u[(size_t)(tb + k) * g.width + c]) : 0.f;
        float A = 1.f, S = 0.f;
#pragma unroll
        for (int k = 0; k < R; ++k) {
            if (tb + k < last) {
                const float la = slope * sigmoid_f(a[k] + rb);
                v[k] = sqrtf(-expm1f(2.0f * la)) * sigmoid_f(v[k] + ib) * uv[k];
                a[k] = expf(la);
                A *= a[k];
                S = fmaf(a[k], S, v[k]);
            }
        }
        float in = carry;
        if (NW > 1) {
            float* pa = rgs_smem + (size_t)p * 2 * NW * X;
            float* ps = pa + (size_t)NW * X;
            pa[w * X + lane] = A;
            ps[w * X + lane] = S;
            __syncthreads();
            float run = carry;
            for (int q = 0; q < NW; ++q) {
                if (q == w) in = run;
                run = fmaf(pa[q * X + lane], run, ps[q * X + lane]);
            }
            carry = run;
        } else {
            carry = fmaf(A, carry, S);
        }
#pragma unroll
        for (int k = 0; k < R; ++k) {
            if (tb + k < last) {
                in = fmaf(a[k], in, v[k]);
                if (live) out[(size_t)(tb + k) * g.width + c] = from_f<T>(in * gelu_tanh_f(yv[k] + yb));
            }
        }
    }
    if (w != 0 || !live) return;
    sp[c] = carry;
    if (g.taps > 1) {
        float* cs = g.conv_state + (int64_t)g.seq_slot[s] * g.slot_stride;
        const float xb = g.x_bias ? g.x_bias[c] : 0.f;
        const int cnt = last - first;
        float keep[B200H_MAX_TAPS];
#pragma unroll
        for (int k = 0; k < B200H_MAX_TAPS - 1; ++k) {
            if (k < g.taps - 1) {
                const int src = cnt + k - (g.taps - 1);
                keep[k] = src >= 0 ? to_f(x[(size_t)(first + src) * g.ld + c]) + xb : cs[(size_t)(src + g.taps - 1) * g.width + c];
            }
        }
#pragma unroll
        for (int k = 0; k < B200H_MAX_TAPS - 1; ++k)
            if (k < g.taps - 1) cs[(size_t)k * g.width + c] = keep[k];
    }
}
