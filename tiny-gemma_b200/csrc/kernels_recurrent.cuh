// Recurrences with one decay per head and token. Per head, with a state S [N][vd]:
//     S <- a_t S + b_t k_t v_t^T,    o_t = S^T q_t
// Two kinds use it; everything between the projections and o_t is fp32:
//   LIN_SSM    (state-space duality) x, B and C come from projections through a short causal convolution with a bias and
//              silu: k = B, q = C (both shared by the heads of a group), v = x; d = softplus(dt + dt_bias),
//              a = exp(-exp(A_log) d), b = d; D_h x_t is added to o_t.
//   LIN_MLSTM  matrix memory with exponential gates: i = cap tanh((.) / cap), f = logsigmoid(cap tanh((.) / cap)), a running
//              maximum m_t = max(f + m_(t-1), i) (from 0), a = exp(f + m_(t-1) - m_t), b = exp(i - m_t); a vector n
//              follows S with v = 1, and o_t is divided by max(|n_t . q_t|, exp(-m_t)) + 1e-6.
// The raw o_t go to an fp32 buffer; norm and gate follow in lin_norm_kernel or in the prologue of the output product.
//
//   lin_token_cta          one token: a CTA per (sequence, head, 32 columns of S)
//   lin_conv_kernel        LIN_SSM: convolution and silu of a portion's x, B, C, padded head by head; log a and b
//   lin_gates_kernel       LIN_MLSTM: log a, b and exp(-m) of a portion's rows
//   lin_scan_kernel        a portion token by token, S in registers: 32-bit states, and portions of a few tokens
//   lin_chunk_*_kernel     portions in chunks of LC = 128 tokens on the tensor cores. With c_t the sum of log a up to t
//                          within the chunk (fp64 sums kept as pairs of floats: strong decays before weak ones lose
//                          nothing) and S_0 the state before it,
//                              o_t = exp(c_t) q_t S_0 + sum_{s<=t} exp(c_t - c_s) b_s (q_t . k_s) v_s
//                              S_1 = exp(c_last) S_0 + sum_s k_s (exp(c_last - c_s) b_s v_s)^T
//                          state: the second sums, all chunks in parallel; scan: S_0 of every chunk, elementwise;
//                          out: o. Operands that are not projections are split into two bf16 terms, except the
//                          weights of (q . k), which enter their product as bf16 (their row sums stay fp32).
#pragma once
#include "kernels_gemm_bf16.cuh"
#include "kernels_rowwise.cuh"
#include "kernels_window_attn.cuh"

namespace tg {

enum LinKind { LIN_NONE = 0, LIN_SSM = 1, LIN_MLSTM = 2 };
constexpr int LC = 128;     // tokens of a chunk
constexpr int LT_COLS = 32; // columns of S per CTA (one token, token by token)

struct LinArgs {
	StepDesc d;
	int kind, H, G, N, vd, Np, vdp;  // G: groups that share q and k; Np, vdp: sizes padded to multiples of 16
	const void *p;           // projections, rows of ldp: raw [x][B][C] at p_x (LIN_SSM); padded q, k, v (LIN_MLSTM)
	int ldp, p_x, p_q, p_k, p_v;
	const float *t;          // fp32 projections, rows of ldt: dt [H], or i [H] and f [H]
	int ldt;
	const float *A_log, *dt_bias, *Dv;   // LIN_SSM [H]
	const float *ib, *fb;                // LIN_MLSTM [H]
	float gate_cap, qscale;
	const float *cw, *cb;    // convolution [taps][C] and bias [C], C = H vd + 2 G N
	int taps;
	float *hist;             // [B][2][taps-1][C] convolution inputs of earlier steps
	void *xc;                // LIN_SSM, portions: [R][ldxc] = [x H vdp][B G Np][C G Np]
	int ldxc;
	const void *rows;        // portions: q, k, v of the rows: xc or p
	int ldr, o_q, o_k, o_v;
	float *S;                // [B][H][N][vdp]
	float *n, *m;            // LIN_MLSTM [B][2][H][N], [B][2][H]: two copies, chosen by parity
	float *la, *b, *em;      // [R][H] log decay, weight of the new term, exp(-m)
	float *o;                // [R][ldo] raw read-outs, head h at h vd
	int ldo;
	// chunks (index: lin_chunk_base)
	float *dS;               // [chunks][H][N][vdp]
	__nv_bfloat16 *Sh, *Sl;  // [chunks][H][Np][vdp] S_0 as two terms
	float *dn, *n0;          // [chunks][H][N]
	float *tot;              // [chunks][H] c_last
	int vsplit;              // out: CTAs that share the columns of a head
	int ready;               // one token: LIN_SSM's convolved rows and log a, b are there already
	int *err;
};

__host__ __device__ inline int lin_channels(const LinArgs &a) { return a.H * a.vd + 2 * a.G * a.N; }
__host__ __device__ inline int lin_chunk_base(int seg_row, int seg) { return seg_row / LC + seg; }

__device__ __forceinline__ float logsigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// (log a, b) of a token; LIN_MLSTM: with f and i instead
__device__ __forceinline__ float2 lin_gate_in(const LinArgs &a, int r, int h) {
	const float *t = a.t + size_t(r) * a.ldt;
	if (a.kind == LIN_SSM) {
		const float dt = softplus_f(t[h] + a.dt_bias[h]);
		return make_float2(-expf(a.A_log[h]) * dt, dt);
	}
	const float c = a.gate_cap;
	return make_float2(logsigmoid_f(c * tanhf((t[a.H + h] + a.fb[h]) / c)), c * tanhf((t[h] + a.ib[h]) / c));
}

// convolution input of channel c at time t of a segment (t < 0: earlier steps)
template <typename PT> __device__ __forceinline__ float lin_conv_in(const LinArgs &a, int row0, int pos, const float *hr, int C, int t, int c) {
	if (t >= 0) return to_f32(reinterpret_cast<const PT *>(a.p)[size_t(row0 + t) * a.ldp + a.p_x + c]);
	return pos + t >= 0 ? hr[size_t(a.taps - 1 + t) * C + c] : 0.0f;
}

// ------------------------------------------------------------------ one token
// 256 threads: 8 across the 32 columns (4 each), 32 down the rows. smem: q[Np] k[Np] v[32] red[9 * 32 + 16]
__host__ __device__ inline size_t lin_token_smem(int Np) { return (size_t(2) * Np + 32 + 9 * 32 + 16) * 4; }
__host__ __device__ inline int lin_token_ctas(int H, int vd) { return H * ((vd + LT_COLS - 1) / LT_COLS); }

template <typename PT> __device__ void lin_token_cta(const LinArgs &a, int r, int item, float *sm) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int tiles = (a.vd + LT_COLS - 1) / LT_COLS, h = item / tiles, tile = item % tiles, per = a.H / a.G, g = h / per, N = a.N;
	const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], pos = a.d.seg_pos[seg], par = a.d.seg_par[seg];
	float *sq = sm, *sk = sq + a.Np, *sv = sk + a.Np, *red = sv + 32;
	const bool fresh = pos == 0;
	const int cl = (tid & 7) * 4, c0 = tile * LT_COLS + cl, rg = tid >> 3;
	float *S = a.S + (size_t(seq) * a.H + h) * N * a.vdp + c0;
	const bool on = c0 < a.vdp;
	constexpr int HOLD = 4;  // rows of the state requested ahead
	float4 st[HOLD];
#pragma unroll
	for (int e = 0; e < HOLD; e++) {
		const int i = rg + 32 * e;
		st[e] = on && !fresh && i < N ? *reinterpret_cast<const float4 *>(S + size_t(i) * a.vdp) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
	}
	const PT *row = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	if (a.kind == LIN_SSM && a.ready) {
		const PT *rr = reinterpret_cast<const PT *>(a.rows) + size_t(r) * a.ldr;
		for (int x = tid; x < N; x += 256) {
			sq[x] = to_f32(rr[a.o_q + g * a.Np + x]);
			sk[x] = to_f32(rr[a.o_k + g * a.Np + x]);
		}
		if (tid < LT_COLS) sv[tid] = tile * LT_COLS + tid < a.vd ? to_f32(rr[a.o_v + h * a.vdp + tile * LT_COLS + tid]) : 0.0f;
	} else if (a.kind == LIN_SSM) {
		const int C = lin_channels(a), H = a.taps - 1;
		float *hb = a.hist + size_t(seq) * 2 * H * C;
		const float *hr = hb + size_t(par) * H * C;
		float *hw = hb + size_t(par ^ 1) * H * C;
		const int nv = min(LT_COLS, a.vd - tile * LT_COLS);
		for (int x = tid; x < 2 * N + LT_COLS; x += 256) {
			if (x >= 2 * N + nv) {
				sv[x - 2 * N] = 0.0f;
				continue;
			}
			const bool isv = x >= 2 * N;
			const int ch = isv ? h * a.vd + tile * LT_COLS + x - 2 * N : a.H * a.vd + (x < N ? g * N + x : (a.G + g) * N + x - N);
			float y = a.cb[ch];
			for (int j = 0; j <= H; j++) {
				const float u = lin_conv_in<PT>(a, r, pos, hr, C, j - H, ch);
				y = fmaf(a.cw[size_t(j) * C + ch], u, y);
				if (j > 0 && (isv || (h % per == 0 && tile == 0))) hw[size_t(j - 1) * C + ch] = u;
			}
			y = silu_f(y);
			(isv ? sv[x - 2 * N] : (x < N ? sk[x] : sq[x - N])) = y;
		}
	} else {
		for (int x = tid; x < N; x += 256) {
			sq[x] = to_f32(row[a.p_q + g * a.Np + x]) * a.qscale;
			sk[x] = to_f32(row[a.p_k + g * a.Np + x]);
		}
		if (tid < LT_COLS) sv[tid] = tile * LT_COLS + tid < a.vd ? to_f32(row[a.p_v + h * a.vdp + tile * LT_COLS + tid]) : 0.0f;
	}
	const float2 gi = a.ready && a.kind == LIN_SSM ? make_float2(a.la[size_t(r) * a.H + h], a.b[size_t(r) * a.H + h]) : lin_gate_in(a, r, h);
	float da, b, mn = 0.0f;
	if (a.kind == LIN_SSM) {
		da = expf(gi.x);
		b = gi.y;
	} else {
		const float m0 = fresh ? 0.0f : a.m[(size_t(seq) * 2 + par) * a.H + h];
		mn = fmaxf(gi.x + m0, gi.y);
		da = expf(gi.x + m0 - mn);
		b = expf(gi.y - mn);
	}
	__syncthreads();
	float4 v = *reinterpret_cast<const float4 *>(sv + cl);
	v.x *= b; v.y *= b; v.z *= b; v.w *= b;
	float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
	auto update = [&](float4 s, int i) {
		const float k = sk[i], q = sq[i];
		s.x = fmaf(da, s.x, k * v.x); s.y = fmaf(da, s.y, k * v.y); s.z = fmaf(da, s.z, k * v.z); s.w = fmaf(da, s.w, k * v.w);
		y.x = fmaf(s.x, q, y.x); y.y = fmaf(s.y, q, y.y); y.z = fmaf(s.z, q, y.z); y.w = fmaf(s.w, q, y.w);
		*reinterpret_cast<float4 *>(S + size_t(i) * a.vdp) = s;
	};
	if (on) {
#pragma unroll
		for (int e = 0; e < HOLD; e++)
			if (rg + 32 * e < N) update(st[e], rg + 32 * e);
		for (int i0 = rg + 32 * HOLD; i0 < N; i0 += 32 * HOLD) {
#pragma unroll
			for (int e = 0; e < HOLD; e++)
				st[e] = !fresh && i0 + 32 * e < N ? *reinterpret_cast<const float4 *>(S + size_t(i0 + 32 * e) * a.vdp) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
			for (int e = 0; e < HOLD; e++)
				if (i0 + 32 * e < N) update(st[e], i0 + 32 * e);
		}
	}
	float den = 0.0f;
	if (a.kind == LIN_MLSTM) {
		const float *nr = a.n + ((size_t(seq) * 2 + par) * a.H + h) * N;
		float *nw = a.n + ((size_t(seq) * 2 + (par ^ 1)) * a.H + h) * N;
		for (int i = tid; i < N; i += 256) {
			const float nn = fmaf(da, fresh ? 0.0f : nr[i], b * sk[i]);
			den = fmaf(nn, sq[i], den);
			if (tile == 0) nw[i] = nn;
		}
		if (tile == 0 && tid == 0) a.m[(size_t(seq) * 2 + (par ^ 1)) * a.H + h] = mn;
		den = warp_sum(den);
	}
#pragma unroll
	for (int x = 8; x < 32; x *= 2) {
		y.x += __shfl_xor_sync(0xffffffffu, y.x, x);
		y.y += __shfl_xor_sync(0xffffffffu, y.y, x);
		y.z += __shfl_xor_sync(0xffffffffu, y.z, x);
		y.w += __shfl_xor_sync(0xffffffffu, y.w, x);
	}
	if (lane < 8) {
		red[warp * 32 + cl] = y.x;
		red[warp * 32 + cl + 1] = y.y;
		red[warp * 32 + cl + 2] = y.z;
		red[warp * 32 + cl + 3] = y.w;
	}
	if (lane == 0) red[8 * 32 + warp] = den;
	__syncthreads();
	if (tid < LT_COLS && tile * LT_COLS + tid < a.vd) {
		float o = 0.0f, dn = 0.0f;
#pragma unroll
		for (int w = 0; w < 8; w++) {
			o += red[w * 32 + tid];
			dn += red[8 * 32 + w];
		}
		if (a.kind == LIN_SSM) o = fmaf(a.Dv[h], sv[tid], o);
		else o /= fmaxf(fabsf(dn), expf(-mn)) + 1e-6f;
		a.o[size_t(r) * a.ldo + h * a.vd + tile * LT_COLS + tid] = o;
	}
}

// ------------------------------------------------------------------ portions: convolution, gates
// V consecutive elements; fast: where the result is rounded to bf16 anyway
template <int V> __device__ __forceinline__ void lin_load(float (&o)[V], const float *p) {
	if constexpr (V == 4) {
		const float4 v = *reinterpret_cast<const float4 *>(p);
		o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
	} else {
		o[0] = p[0];
	}
}
template <int V> __device__ __forceinline__ void lin_load(float (&o)[V], const __nv_bfloat16 *p) {
	if constexpr (V == 4) {
		const uint2 u = *reinterpret_cast<const uint2 *>(p);
		o[0] = bf16_lo(u.x); o[1] = bf16_hi(u.x); o[2] = bf16_lo(u.y); o[3] = bf16_hi(u.y);
	} else {
		o[0] = __bfloat162float(p[0]);
	}
}
template <int V, typename T> __device__ __forceinline__ void lin_store(T *p, const float (&o)[V]) {
	if constexpr (V == 4) store4<T>(p, make_float4(o[0], o[1], o[2], o[3]));
	else p[0] = from_f32<T>(o[0]);
}
template <typename T> __device__ __forceinline__ float lin_sigmoid(float z) {
	return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-z)) : sigmoid_f(z);
}

// grid (ceil(R / rows), ceil(ldxc / (128 V)) + 1), 128 threads, rows <= LV_ROWS: a thread walks the rows of V (padded)
// columns, the window in registers. V = 4 if groups of four columns are channels that follow each other. The last blockIdx.y forms the
// rows' log a and b.
constexpr int LV_ROWS = 16;
template <typename PT, int MT, int V> __global__ void __launch_bounds__(128) lin_conv_kernel(LinArgs a, int R, int rows) {
	pdl_trigger();
	pdl_wait();
	__shared__ int seg_s[LV_ROWS];
	const int tid = threadIdx.x, r0 = blockIdx.x * rows, nr = min(rows, R - r0);
	if (blockIdx.y + 1 == gridDim.y) {
		for (int x = tid; x < nr * a.H; x += 128) {
			const int r = r0 + x / a.H, h = x % a.H;
			const float2 g = lin_gate_in(a, r, h);
			a.la[size_t(r) * a.H + h] = g.x;
			a.b[size_t(r) * a.H + h] = g.y;
		}
		return;
	}
	if (tid < nr) seg_s[tid] = a.d.row_seg[r0 + tid];
	__syncthreads();
	const int col = V * (blockIdx.y * 128 + tid);
	if (col >= a.ldxc) return;
	const int C = lin_channels(a), H = a.taps - 1;
	const int xw = a.H * a.vdp, bw = a.G * a.Np;
	int ch;  // the raw channel, or -1 for padding
	if (col < xw) ch = col % a.vdp < a.vd ? col / a.vdp * a.vd + col % a.vdp : -1;
	else {
		const int c = (col - xw) % bw, which = (col - xw) / bw;
		ch = c % a.Np < a.N && which < 2 ? a.H * a.vd + which * a.G * a.N + c / a.Np * a.N + c % a.Np : -1;
	}
	PT *out = reinterpret_cast<PT *>(a.xc) + size_t(r0) * a.ldxc + col;
	if (ch < 0) {
		const float none[V] = {};
		for (int i = 0; i < nr; i++) lin_store<V, PT>(out + size_t(i) * a.ldxc, none);
		return;
	}
	const PT *in = reinterpret_cast<const PT *>(a.p) + size_t(r0) * a.ldp + a.p_x + ch;
	float bias[V], cf[MT][V], win[MT][V];
	lin_load<V>(bias, a.cb + ch);
#pragma unroll
	for (int j = 0; j < MT; j++) {
#pragma unroll
		for (int e = 0; e < V; e++) cf[j][e] = win[j][e] = 0.0f;
		if (j >= MT - a.taps) lin_load<V>(cf[j], a.cw + size_t(j - (MT - a.taps)) * C + ch);
	}
	int seg = -1, row0 = 0, len = 0;
	float *hw = nullptr;
	// the rows before the first one are plain rows of its segment in all but the first few rows of a segment
	const int before = r0 - a.d.seg_row[seg_s[0]];
	if (before >= H) {
		seg = seg_s[0];
		row0 = a.d.seg_row[seg];
		len = a.d.seg_len[seg];
		hw = a.hist + (size_t(a.d.seg_seq[seg]) * 2 + (a.d.seg_par[seg] ^ 1)) * H * C;
#pragma unroll
		for (int j = 0; j < MT; j++)
			if (MT - j <= H) lin_load<V>(win[j], in - ptrdiff_t(MT - j) * a.ldp);
	}
#pragma unroll 1
	for (int i0 = 0; i0 < nr; i0 += 4) {
		float x[4][V];
#pragma unroll
		for (int u = 0; u < 4; u++) {
#pragma unroll
			for (int e = 0; e < V; e++) x[u][e] = 0.0f;
			if (i0 + u < nr) lin_load<V>(x[u], in + size_t(i0 + u) * a.ldp);
		}
#pragma unroll
		for (int u = 0; u < 4; u++) {
			const int i = i0 + u, r = r0 + i;
			if (i >= nr) break;
			if (seg_s[i] != seg) {
				seg = seg_s[i];
				row0 = a.d.seg_row[seg];
				len = a.d.seg_len[seg];
				const int pos = a.d.seg_pos[seg], t = r - row0;
				float *hb = a.hist + size_t(a.d.seg_seq[seg]) * 2 * H * C;
				const float *hr = hb + size_t(a.d.seg_par[seg]) * H * C;
				hw = hb + size_t(a.d.seg_par[seg] ^ 1) * H * C;
#pragma unroll
				for (int j = 0; j < MT; j++)
#pragma unroll
					for (int e = 0; e < V; e++) win[j][e] = MT - j <= H ? lin_conv_in<PT>(a, row0, pos, hr, C, t - (MT - j), ch + e) : 0.0f;
				if (t == 0)  // inputs before this segment that stay relevant
					for (int q = 0; q < H; q++)
						if (len - H + q < 0)
							for (int e = 0; e < V; e++) hw[size_t(q) * C + ch + e] = lin_conv_in<PT>(a, row0, pos, hr, C, len - H + q, ch + e);
			}
			float y[V];
#pragma unroll
			for (int e = 0; e < V; e++) {
				y[e] = bias[e];
#pragma unroll
				for (int j = 0; j < MT; j++) {
					win[j][e] = j + 1 < MT ? win[j + 1][e] : x[u][e];
					y[e] = fmaf(cf[j][e], win[j][e], y[e]);
				}
				y[e] = sizeof(PT) == 2 ? swish_fast(y[e], y[e]) : silu_f(y[e]);
			}
			lin_store<V, PT>(out + size_t(i) * a.ldxc, y);
			const int q = (r - row0) - (len - H);
			if (q >= 0) lin_store<V, float>(hw + size_t(q) * C + ch, x[u]);
		}
	}
}

// LIN_MLSTM: log a, b and exp(-m). grid (H, segments), LG_THREADS; a scan of (f, i) pairs, (F1, M1)(F2, M2) =
// (F1 + F2, max(M1 + F2, M2)), four tokens per thread and round
constexpr int LG_THREADS = 1024;
static __global__ void __launch_bounds__(LG_THREADS) lin_gates_kernel(LinArgs a) {
	pdl_trigger();
	pdl_wait();
	__shared__ float sF[LG_THREADS / 32], sM[LG_THREADS / 32];
	const int h = blockIdx.x, seg = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg];
	const int seq = a.d.seg_seq[seg], par = a.d.seg_par[seg];
	float m0 = a.d.seg_pos[seg] == 0 ? 0.0f : a.m[(size_t(seq) * 2 + par) * a.H + h];
	for (int t0 = 0; t0 < len; t0 += 4 * LG_THREADS) {
		float f[4], in[4];
		float F = 0.0f, M = -INFINITY;
#pragma unroll
		for (int j = 0; j < 4; j++) {
			const int t = t0 + 4 * tid + j;
			const float2 g = t < len ? lin_gate_in(a, row0 + t, h) : make_float2(0.0f, -INFINITY);
			f[j] = g.x;
			in[j] = g.y;
			M = fmaxf(M + f[j], in[j]);
			F += f[j];
		}
#pragma unroll
		for (int x = 1; x < 32; x *= 2) {
			const float Fp = __shfl_up_sync(0xffffffffu, F, x), Mp = __shfl_up_sync(0xffffffffu, M, x);
			if (lane >= x) {
				M = fmaxf(Mp + F, M);
				F += Fp;
			}
		}
		if (lane == 31) {
			sF[warp] = F;
			sM[warp] = M;
		}
		// what precedes this thread: the carry, the warps before, the lanes before
		float Fl = __shfl_up_sync(0xffffffffu, F, 1), Ml = __shfl_up_sync(0xffffffffu, M, 1);
		__syncthreads();
		float m = m0;
		for (int w = 0; w < warp; w++) m = fmaxf(m + sF[w], sM[w]);
		if (lane > 0) m = fmaxf(m + Fl, Ml);
#pragma unroll
		for (int j = 0; j < 4; j++) {
			const int t = t0 + 4 * tid + j;
			if (t < len) {
				const float mn = fmaxf(f[j] + m, in[j]);
				const size_t at = size_t(row0 + t) * a.H + h;
				a.la[at] = f[j] + (m - mn);
				a.b[at] = expf(in[j] - mn);
				a.em[at] = expf(-mn);
				m = mn;
			}
		}
		for (int w = 0; w < LG_THREADS / 32; w++) m0 = fmaxf(m0 + sF[w], sM[w]);
		// (the carried maximum is the one the last token stored)
		__syncthreads();
		if (t0 + 4 * LG_THREADS >= len) {
			if (tid == (len - 1 - t0) / 4) a.m[(size_t(seq) * 2 + (par ^ 1)) * a.H + h] = m;
		}
	}
}

// ------------------------------------------------------------------ portions, token by token
// grid (column tiles, H, segments), 256 threads as in lin_token_cta; RPT rows of S per thread
template <typename PT, int RPT> __global__ void __launch_bounds__(256) lin_scan_kernel(LinArgs a) {
	pdl_trigger();
	pdl_wait();
	__shared__ float red[2][8][36];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, tile = blockIdx.x, h = blockIdx.y, seg = blockIdx.z;
	const int N = a.N, g = h / (a.H / a.G), seq = a.d.seg_seq[seg], par = a.d.seg_par[seg], pos = a.d.seg_pos[seg], len = a.d.seg_len[seg], row0 = a.d.seg_row[seg];
	const int cl = (tid & 7) * 4, c0 = tile * LT_COLS + cl, rg = tid >> 3;
	const bool on = c0 < a.vdp, lstm = a.kind == LIN_MLSTM;
	float *S = a.S + (size_t(seq) * a.H + h) * N * a.vdp + c0;
	const float *nr = a.n + ((size_t(seq) * 2 + par) * a.H + h) * N;
	float4 st[RPT];
	float nn[RPT];
#pragma unroll
	for (int e = 0; e < RPT; e++) {
		const int i = rg + 32 * e;
		st[e] = on && pos > 0 && i < N ? *reinterpret_cast<const float4 *>(S + size_t(i) * a.vdp) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
		nn[e] = lstm && pos > 0 && i < N ? nr[i] : 0.0f;
	}
	const PT *base = reinterpret_cast<const PT *>(a.rows);
	float q[RPT], k[RPT], la, b;
	float v[4];
	auto load = [&](int t) {
		const PT *row = base + size_t(row0 + t) * a.ldr;
#pragma unroll
		for (int e = 0; e < RPT; e++) {
			const int i = rg + 32 * e;
			q[e] = i < N ? to_f32(row[a.o_q + g * a.Np + i]) : 0.0f;
			k[e] = i < N ? to_f32(row[a.o_k + g * a.Np + i]) : 0.0f;
		}
#pragma unroll
		for (int e = 0; e < 4; e++) v[e] = on ? to_f32(row[a.o_v + h * a.vdp + c0 + e]) : 0.0f;
		la = a.la[size_t(row0 + t) * a.H + h];
		b = a.b[size_t(row0 + t) * a.H + h];
	};
	load(0);
	for (int t = 0; t < len; t++) {
		const float da = expf(la), v0 = v[0] * b, v1 = v[1] * b, v2 = v[2] * b, v3 = v[3] * b;
		float y0 = 0.0f, y1 = 0.0f, y2 = 0.0f, y3 = 0.0f, den = 0.0f;
#pragma unroll
		for (int e = 0; e < RPT; e++) {
			st[e].x = fmaf(da, st[e].x, k[e] * v0); st[e].y = fmaf(da, st[e].y, k[e] * v1);
			st[e].z = fmaf(da, st[e].z, k[e] * v2); st[e].w = fmaf(da, st[e].w, k[e] * v3);
			nn[e] = fmaf(da, nn[e], b * k[e]);
			y0 = fmaf(st[e].x, q[e], y0); y1 = fmaf(st[e].y, q[e], y1); y2 = fmaf(st[e].z, q[e], y2); y3 = fmaf(st[e].w, q[e], y3);
			den = fmaf(nn[e], q[e], den);
		}
		if (t + 1 < len) load(t + 1);
#pragma unroll
		for (int x = 8; x < 32; x *= 2) {
			y0 += __shfl_xor_sync(0xffffffffu, y0, x);
			y1 += __shfl_xor_sync(0xffffffffu, y1, x);
			y2 += __shfl_xor_sync(0xffffffffu, y2, x);
			y3 += __shfl_xor_sync(0xffffffffu, y3, x);
			den += __shfl_xor_sync(0xffffffffu, den, x);
		}
		float *rd = red[t & 1][warp];
		if (lane < 8) {
			rd[cl] = y0; rd[cl + 1] = y1; rd[cl + 2] = y2; rd[cl + 3] = y3;
		}
		if (lane == 0) rd[32] = den;
		__syncthreads();
		if (tid < LT_COLS && tile * LT_COLS + tid < a.vd) {
			const int c = tile * LT_COLS + tid;
			float o = 0.0f, dn = 0.0f;
#pragma unroll
			for (int w = 0; w < 8; w++) {
				o += red[t & 1][w][tid];
				dn += red[t & 1][w][32];
			}
			const int r = row0 + t;
			if (lstm) o = o * a.qscale / (fmaxf(fabsf(dn * a.qscale), a.em[size_t(r) * a.H + h]) + 1e-6f);
			else o = fmaf(a.Dv[h], to_f32(base[size_t(r) * a.ldr + a.o_v + h * a.vdp + c]), o);
			a.o[size_t(r) * a.ldo + h * a.vd + c] = o;
		}
	}
	float *nw = a.n + ((size_t(seq) * 2 + (par ^ 1)) * a.H + h) * N;
#pragma unroll
	for (int e = 0; e < RPT; e++) {
		const int i = rg + 32 * e;
		if (on && i < N) *reinterpret_cast<float4 *>(S + size_t(i) * a.vdp) = st[e];
		if (lstm && tile == 0 && (tid & 7) == 0 && i < N) nw[i] = nn[e];
	}
}

// ------------------------------------------------------------------ chunks on the tensor cores
// 64 columns x 128 rows of bf16 with the 128-byte swizzle are 16 KB; 16 bytes (8 columns) of a row:
__device__ __forceinline__ uint32_t lin_sw(int row, int c8) { return uint32_t((c8 >> 3) * 16384 + row * 128 + (((c8 & 7) ^ (row & 7)) << 4)); }
// a wait for copies that the CTA started: should it run out, the copies get as long once more before the CTA goes on to its end
__device__ __forceinline__ bool lin_wait_copies(uint64_t *bar, uint32_t parity, int *err) {
	if (tc_wait(bar, parity, err)) return true;
	tc_wait(bar, parity, err);
	return false;
}
__device__ __forceinline__ uint4 lin_ld16(const uint8_t *p) { return *reinterpret_cast<const uint4 *>(p); }

// c_t of 128 tokens in powers of two, as pairs of floats, into smem (threads 0..127; ends with a CTA barrier)
__device__ __forceinline__ void lin_cumulate(float la, float *ch, float *cl, double *part) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	double s = tid < LC ? double(la) * 1.4426950408889634 : 0.0;
	if (tid < LC) {
#pragma unroll
		for (int x = 1; x < 32; x *= 2) {
			const double u = __shfl_up_sync(0xffffffffu, s, x);
			if (lane >= x) s += u;
		}
		if (lane == 31) part[warp] = s;
	}
	__syncthreads();
	if (tid < LC) {
		for (int w = 0; w < warp; w++) s += part[w];
		const float hi = float(s);
		ch[tid] = hi;
		cl[tid] = float(s - double(hi));
	}
	__syncthreads();
}

// ---- the chunks' own contributions to the state: grid (chunks of the longest segment, H x column tiles of 64, segments)
__host__ __device__ inline int lin_kch(int Np) { return (Np + 63) / 64; }
__host__ __device__ inline size_t lin_state_smem(int Np) { return size_t((lin_kch(Np) + 1) / 2 * 2 + 2) * 16384 + 1024; }

static __global__ void __launch_bounds__(256) lin_chunk_state_kernel(const __grid_constant__ CUtensorMap rmap, LinArgs a) {
	pdl_trigger();
	extern __shared__ uint8_t lc_raw[];
	uint8_t *smem = reinterpret_cast<uint8_t *>((uintptr_t(lc_raw) + 1023) & ~uintptr_t(1023));
	__shared__ uint64_t k_bar, d_bar;
	__shared__ uint32_t tmem_base_s;
	__shared__ float ch[LC], cl[LC], sw[LC];
	__shared__ double part[4];
	const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const int kch = lin_kch(a.Np), kchp = (kch + 1) / 2 * 2, mblocks = kchp / 2;
	const uint32_t ncols = mblocks <= 1 ? 64 : 128;
	uint8_t *wh = smem + kchp * 16384, *wl = wh + 16384;
	if (tid == 0) {
		mbar_init(&k_bar, 1);
		mbar_init(&d_bar, 1);
		asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
	}
	pdl_wait();  // (before the allocation: a CTA that holds TMEM waits for no earlier kernel)
	if (warp == 0) {
		asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(ncols) : "memory");
		asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem = tmem_base_s;
	const int vt = (a.vdp + 63) / 64, h = blockIdx.y / vt, tile = blockIdx.y % vt, seg = blockIdx.z, g = h / (a.H / a.G);
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], t0 = blockIdx.x * LC;
	if (t0 < len) {
		const int n = min(LC, len - t0), cols = min(64, a.vdp - 64 * tile);
		const size_t chunk = size_t(lin_chunk_base(row0, seg)) + blockIdx.x, hc = chunk * a.H + h;
		if (tid == 0) {
			mbar_expect_tx(&k_bar, uint32_t(kch) * 16384);
			for (int c = 0; c < kch; c++) tma_load_2d(smem + c * 16384, &rmap, a.o_k + g * a.Np + 64 * c, row0 + t0, &k_bar);
		}
		const float b = tid < n ? a.b[size_t(row0 + t0 + tid) * a.H + h] : 0.0f;
		const __nv_bfloat16 *vb = reinterpret_cast<const __nv_bfloat16 *>(a.rows) + size_t(row0 + t0) * a.ldr + a.o_v + h * a.vdp + 64 * tile;
		const int c8n = cols / 8;
		uint4 vr[4];  // 16 bytes of V per thread and round; at most four rounds
#pragma unroll
		for (int e = 0; e < 4; e++) {
			const int x = tid + 256 * e, s = x / c8n;
			vr[e] = s < n ? *reinterpret_cast<const uint4 *>(vb + size_t(s) * a.ldr + 8 * (x % c8n)) : make_uint4(0, 0, 0, 0);
		}
		lin_cumulate(tid < n ? a.la[size_t(row0 + t0 + tid) * a.H + h] : 0.0f, ch, cl, part);
		if (tid < LC) sw[tid] = b * exp2f((ch[LC - 1] - ch[tid]) + (cl[LC - 1] - cl[tid]));
		if (tid == 0 && tile == 0) a.tot[hc] = ch[LC - 1] + cl[LC - 1];
		__syncthreads();
#pragma unroll
		for (int r = 0; r < 4; r++) {
			const int x = tid + 256 * r, s = x / c8n, c8 = x % c8n;
			if (s >= LC) break;
			const uint4 u = vr[r];
			const float w = sw[s];
			const uint32_t in[4] = {u.x, u.y, u.z, u.w};
			uint32_t hi[4], lo[4];
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const float p = bf16_lo(in[e]) * w, q = bf16_hi(in[e]) * w;
				hi[e] = pack_bf16(p, q);
				lo[e] = pack_bf16(p - bf16_lo(hi[e]), q - bf16_hi(hi[e]));
			}
			*reinterpret_cast<uint4 *>(wh + lin_sw(s, c8)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
			*reinterpret_cast<uint4 *>(wl + lin_sw(s, c8)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
		}
		fence_proxy_async();
		__syncthreads();
		bool ok = true;
		if (tid == 0) {
			ok = lin_wait_copies(&k_bar, 0, a.err);
			if (ok) {
				tc_fence_after();
				const uint32_t idesc = tc_idesc_bf16(cols, 1) | (1u << 15);  // both operands MN-major
				const uint32_t ka = smem_u32(smem), wa = smem_u32(wh), wb = smem_u32(wl);
				for (int mb = 0; mb < mblocks; mb++)
					for (int j = 0; j < 2 * LC / 16; j++) {
						const int kk = j & 7;
						tc_mma(tmem + uint32_t(mb * 64), tc_sw128_desc(ka + mb * 32768 + kk * 2048, 16384, 1024), tc_sw128_desc((j < 8 ? wa : wb) + kk * 2048, 16384, 1024), idesc,
						       j > 0 ? 1u : 0u);
					}
				tc_commit(&d_bar);
			}
		}
		if (a.kind == LIN_MLSTM && tile == 0) {
			const bool okk = tc_wait(&k_bar, 0, a.err);
			for (int c = tid; c < a.N && okk; c += 256) {
				float s = 0.0f;
				for (int t = 0; t < n; t++) {
					const __nv_bfloat16 *kp = reinterpret_cast<const __nv_bfloat16 *>(smem + lin_sw(t, c >> 3)) + (c & 7);
					s = fmaf(sw[t], __bfloat162float(*kp), s);
				}
				a.dn[hc * a.N + c] = s;
			}
		}
		__syncwarp();
		// (a failed k_bar wait leaves d_bar uncommitted: this wait runs out too)
		ok = __all_sync(0xffffffffu, tc_wait(&d_bar, 0, a.err)) != 0;
		if (ok) {
			tc_fence_after();
			const int quad = warp & 3, half = warp >> 2;
			for (int mb = 0; mb < mblocks; mb++) {
				const int i = mb * 128 + quad * 32 + lane;
				float *dst = a.dS + (hc * a.N + i) * a.vdp + 64 * tile;
				for (int c = 16 * half; c < cols; c += 32) {
					uint32_t o[16];
					wt_ld16(tmem + (uint32_t(quad * 32) << 16) + uint32_t(mb * 64 + c), o);
					if (i < a.N) {
#pragma unroll
						for (int q = 0; q < 4; q++) *reinterpret_cast<uint4 *>(dst + c + 4 * q) = make_uint4(o[4 * q], o[4 * q + 1], o[4 * q + 2], o[4 * q + 3]);
					}
				}
			}
		}
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(ncols));
}

// ---- S_0 of every chunk, and the state after the last: a thread owns four columns of a row (or an element of n)
// grid (ceil(items / 256), segments); items = H N vdp / 4, then H N of n (LIN_MLSTM)
static __global__ void __launch_bounds__(256) lin_chunk_scan_kernel(LinArgs a) {
	pdl_trigger();
	pdl_wait();
	const int seg = blockIdx.y, v4 = a.vdp / 4, items = a.H * a.N * v4;
	const int len = a.d.seg_len[seg], seq = a.d.seg_seq[seg], par = a.d.seg_par[seg], nc = (len + LC - 1) / LC;
	const bool fresh = a.d.seg_pos[seg] == 0;
	const size_t chunk0 = lin_chunk_base(a.d.seg_row[seg], seg);
	int x = blockIdx.x * 256 + threadIdx.x;
	if (x < items) {
		const int h = x / (a.N * v4), i = x / v4 % a.N, c = 4 * (x % v4);
		float *Sg = a.S + ((size_t(seq) * a.H + h) * a.N + i) * a.vdp + c;
		float4 S = fresh ? make_float4(0.0f, 0.0f, 0.0f, 0.0f) : *reinterpret_cast<const float4 *>(Sg);
		for (int k0 = 0; k0 < nc; k0 += 4) {
			float4 d[4];
			float A[4];
#pragma unroll
			for (int u = 0; u < 4; u++) {
				const size_t hc = (chunk0 + k0 + u) * a.H + h;
				d[u] = k0 + u < nc ? *reinterpret_cast<const float4 *>(a.dS + (hc * a.N + i) * a.vdp + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
				A[u] = k0 + u < nc ? a.tot[hc] : 0.0f;
			}
#pragma unroll
			for (int u = 0; u < 4; u++) {
				if (k0 + u >= nc) break;
				const size_t at = (((chunk0 + k0 + u) * a.H + h) * a.Np + i) * a.vdp + c;
				const uint32_t h0 = pack_bf16(S.x, S.y), h1 = pack_bf16(S.z, S.w);
				*reinterpret_cast<uint2 *>(a.Sh + at) = make_uint2(h0, h1);
				*reinterpret_cast<uint2 *>(a.Sl + at) =
				    make_uint2(pack_bf16(S.x - bf16_lo(h0), S.y - bf16_hi(h0)), pack_bf16(S.z - bf16_lo(h1), S.w - bf16_hi(h1)));
				const float e = exp2f(A[u]);
				S.x = fmaf(e, S.x, d[u].x); S.y = fmaf(e, S.y, d[u].y); S.z = fmaf(e, S.z, d[u].z); S.w = fmaf(e, S.w, d[u].w);
			}
		}
		*reinterpret_cast<float4 *>(Sg) = S;
		return;
	}
	x -= items;
	if (a.kind != LIN_MLSTM || x >= a.H * a.N) return;
	const int h = x / a.N, i = x % a.N;
	float s = fresh ? 0.0f : a.n[((size_t(seq) * 2 + par) * a.H + h) * a.N + i];
	for (int k = 0; k < nc; k++) {
		const size_t hc = (chunk0 + k) * a.H + h;
		a.n0[hc * a.N + i] = s;
		s = fmaf(exp2f(a.tot[hc]), s, a.dn[hc * a.N + i]);
	}
	a.n[((size_t(seq) * 2 + (par ^ 1)) * a.H + h) * a.N + i] = s;
}

// ---- read-outs: grid (chunks of the longest segment, H x vsplit, segments), 256 threads, two per query row.
// TMEM: scores in columns 0..127, their bf16 weights over columns 0..63, q S_0 in 128..191, weights x V in 192..255.
// Shared memory: Q, then K, later S_0's two terms in K's place, then V tiles of 64 columns.
__host__ __device__ inline size_t lin_out_smem(int Np) {
	const size_t k = size_t(lin_kch(Np)) * 16384, s = size_t(2) * Np * 128;
	return k + (k > s ? k : s) + 16384 + 1024;
}
static __global__ void __launch_bounds__(256, 2) lin_chunk_out_kernel(const __grid_constant__ CUtensorMap rmap, const __grid_constant__ CUtensorMap shmap,
                                                                     const __grid_constant__ CUtensorMap slmap, LinArgs a) {
	pdl_trigger();
	extern __shared__ uint8_t lc_raw[];
	uint8_t *smem = reinterpret_cast<uint8_t *>((uintptr_t(lc_raw) + 1023) & ~uintptr_t(1023));
	__shared__ uint64_t qk_bar, s_bar, sv_bar, o_bar;
	__shared__ uint32_t tmem_base_s;
	__shared__ float ch[LC], cl[LC], sb[LC], xch[2][LC], den_s[LC];
	__shared__ double part[4];
	const int tid = threadIdx.x, warp = tid >> 5;
	const int kch = lin_kch(a.Np);
	uint8_t *sQ = smem, *sK = sQ + kch * 16384, *sS = sK;
	const uint32_t kbytes = uint32_t(kch) * 16384, sbytes = uint32_t(a.Np) * 128;
	uint8_t *sV = sK + (kbytes > 2 * sbytes ? kbytes : 2 * sbytes);
	if (tid == 0) {
		mbar_init(&qk_bar, 1);
		mbar_init(&s_bar, 1);
		mbar_init(&sv_bar, 1);
		mbar_init(&o_bar, 1);
		asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
	}
	pdl_wait();  // (before the allocation: a CTA that holds TMEM waits for no earlier kernel)
	if (warp == 0) {
		asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(256) : "memory");
		asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem = tmem_base_s;
	const int h = blockIdx.y / a.vsplit, vs = blockIdx.y % a.vsplit, seg = blockIdx.z, g = h / (a.H / a.G);
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], t0 = blockIdx.x * LC;
	const int tiles = (a.vdp + 63) / 64, share = (tiles + a.vsplit - 1) / a.vsplit, tl0 = vs * share, tl1 = min(tiles, tl0 + share);
	if (t0 < len && tl0 < tl1) {
		const int n = min(LC, len - t0);
		const size_t hc = (size_t(lin_chunk_base(row0, seg)) + blockIdx.x) * a.H + h;
		// V of a column tile and S_0 under the same 64 columns
		auto fetch_v = [&](int tl) { tma_load_2d(sV, &rmap, a.o_v + h * a.vdp + 64 * tl, row0 + t0, &sv_bar); };
		auto fetch_s = [&](int tl) {
			tma_load_2d(sS, &shmap, 64 * tl, int(hc) * a.Np, &sv_bar);  // (boxes of Np rows)
			tma_load_2d(sS + sbytes, &slmap, 64 * tl, int(hc) * a.Np, &sv_bar);
		};
		const uint32_t svbytes = 16384 + 2 * sbytes;
		if (tid == 0) {
			mbar_expect_tx(&qk_bar, 2 * kbytes);
			for (int c = 0; c < kch; c++) {
				tma_load_2d(sQ + c * 16384, &rmap, a.o_q + g * a.Np + 64 * c, row0 + t0, &qk_bar);
				tma_load_2d(sK + c * 16384, &rmap, a.o_k + g * a.Np + 64 * c, row0 + t0, &qk_bar);
			}
			mbar_expect_tx(&sv_bar, svbytes);
			fetch_v(tl0);
		}
		if (tid < LC) sb[tid] = tid < n ? a.b[size_t(row0 + t0 + tid) * a.H + h] : 0.0f;
		lin_cumulate(tid < n ? a.la[size_t(row0 + t0 + tid) * a.H + h] : 0.0f, ch, cl, part);
		const uint32_t qa = smem_u32(sQ), ka = smem_u32(sK), sa = smem_u32(sS), va = smem_u32(sV);
		if (tid == 0) {
			if (lin_wait_copies(&qk_bar, 0, a.err)) {
				tc_fence_after();
				const uint32_t idesc = tc_idesc_bf16(LC, 0);
				for (int j = 0; j < a.Np / 16; j++)
					tc_mma(tmem, tc_sw128_desc(qa + (j >> 2) * 16384 + (j & 3) * 32, 16, 1024), tc_sw128_desc(ka + (j >> 2) * 16384 + (j & 3) * 32, 16, 1024), idesc, j > 0 ? 1u : 0u);
			}
			tc_commit(&s_bar);
		}
		__syncwarp();
		const int row = tid & 127, half = tid >> 7, quad = warp & 3;
		const uint32_t lane_addr = uint32_t(quad * 32) << 16;
		bool ok = __all_sync(0xffffffffu, tc_wait(&s_bar, 0, a.err)) != 0;
		tc_fence_after();
		if (tid == 0) fetch_s(tl0);  // (K has been read)
		float sum = 0.0f;
		{
			uint32_t w[32];
			const float th = ch[row], tl = cl[row];
			const int last = min(row, n - 1) - 64 * half;  // columns of this half up to `last` are visible
#pragma unroll
			for (int e = 0; e < 2; e++) {
				if (64 * half + 32 * e > 32 * quad + 31) {  // (the whole warp: nothing of this block is visible)
#pragma unroll
					for (int c = 0; c < 16; c++) w[16 * e + c] = 0;
					continue;
				}
				uint32_t ra[32];
				tc_ld32(tmem + lane_addr + uint32_t(64 * half + 32 * e), ra);
				asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
				for (int c = 0; c < 32; c += 2) {
					const int s = 64 * half + 32 * e + c;
					const float d0 = (th - ch[s]) + (tl - cl[s]), d1 = (th - ch[s + 1]) + (tl - cl[s + 1]);
					const float p0 = 32 * e + c <= last ? __uint_as_float(ra[c]) * ex2_f(d0) * sb[s] : 0.0f;
					const float p1 = 32 * e + c + 1 <= last ? __uint_as_float(ra[c + 1]) * ex2_f(d1) * sb[s + 1] : 0.0f;
					sum += p0 + p1;
					w[16 * e + c / 2] = pack_bf16(p0, p1);
				}
			}
			xch[half][row] = sum;
			asm volatile("bar.sync %0, 64;" ::"r"(1 + quad) : "memory");  // both halves of a row have been read
			tc_st32(tmem + lane_addr + uint32_t(32 * half), w);
			asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
			tc_fence_before();
		}
		const float ec = exp2f(ch[row] + cl[row]);
		float f = a.qscale;
		if (a.kind == LIN_MLSTM) {  // n_t . q_t, half of the key columns per thread
			float s = 0.0f;
			const int c8h = (a.Np / 8 + 1) / 2;
			for (int c8 = half * c8h; c8 < min(a.Np / 8, (half + 1) * c8h); c8++) {
				const uint4 u = lin_ld16(sQ + lin_sw(row, c8));
				const uint32_t in[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
				for (int e = 0; e < 4; e++) {
					const int c = 8 * c8 + 2 * e;
					if (c < a.N) s = fmaf(bf16_lo(in[e]), a.n0[hc * a.N + c], s);
					if (c + 1 < a.N) s = fmaf(bf16_hi(in[e]), a.n0[hc * a.N + c + 1], s);
				}
			}
			sum += xch[half ^ 1][row];
			if (half == 0) den_s[row] = s;
			asm volatile("bar.sync %0, 64;" ::"r"(1 + quad) : "memory");
			if (half == 1) {
				s += den_s[row];
				den_s[row] = s;
			}
			asm volatile("bar.sync %0, 64;" ::"r"(1 + quad) : "memory");
			const float den = a.qscale * fmaf(ec, den_s[row], sum);
			const float em = row < n ? a.em[size_t(row0 + t0 + row) * a.H + h] : 1.0f;
			f = a.qscale / (fmaxf(fabsf(den), em) + 1e-6f);
		}
		const float Dh = a.kind == LIN_SSM ? a.Dv[h] : 0.0f;
		__syncthreads();
		for (int tl = tl0; tl < tl1; tl++) {
			const int cols = min(64, a.vdp - 64 * tl), par = (tl - tl0) & 1;
			if (tid == 0) {
				if (lin_wait_copies(&sv_bar, par, a.err)) {
					tc_fence_after();
					const uint32_t idesc = tc_idesc_bf16(cols, 1);
					for (int j = 0; j < a.Np / 16; j++)
						for (int e = 0; e < 2; e++)
							tc_mma(tmem + 128, tc_sw128_desc(qa + (j >> 2) * 16384 + (j & 3) * 32, 16, 1024), tc_sw128_desc(sa + e * sbytes + j * 2048, 16384, 1024), idesc,
							       j + e > 0 ? 1u : 0u);
					for (int j = 0; j < LC / 16; j++)
						tc_mma_ta(tmem + 192, tmem + uint32_t(j * 8), tc_sw128_desc(va + j * 2048, 16384, 1024), idesc, j > 0 ? 1u : 0u);
				}
				tc_commit(&o_bar);
			}
			__syncwarp();
			ok = __all_sync(0xffffffffu, tc_wait(&o_bar, par, a.err)) != 0 && ok;
			tc_fence_after();
			float *out = a.o + size_t(row0 + t0 + row) * a.ldo + h * a.vd + 64 * tl;
			const int left = a.vd - 64 * tl;
			for (int c = 16 * half; c < cols; c += 32) {
				uint32_t o1[16], o2[16];
				wt_ld16(tmem + lane_addr + uint32_t(128 + c), o1);
				wt_ld16(tmem + lane_addr + uint32_t(192 + c), o2);
				if (row < n && ok) {
					const uint4 u0 = lin_ld16(sV + lin_sw(row, c >> 3)), u1 = lin_ld16(sV + lin_sw(row, (c >> 3) + 1));
					const uint32_t in[8] = {u0.x, u0.y, u0.z, u0.w, u1.x, u1.y, u1.z, u1.w};
					float y[16];
#pragma unroll
					for (int q = 0; q < 16; q++) {
						const float v = (q & 1) ? bf16_hi(in[q >> 1]) : bf16_lo(in[q >> 1]);
						y[q] = fmaf(Dh, v, f * fmaf(ec, __uint_as_float(o1[q]), __uint_as_float(o2[q])));
					}
					if (left >= c + 16 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
#pragma unroll
						for (int q = 0; q < 4; q++) *reinterpret_cast<float4 *>(out + c + 4 * q) = make_float4(y[4 * q], y[4 * q + 1], y[4 * q + 2], y[4 * q + 3]);
					} else {
#pragma unroll
						for (int q = 0; q < 16; q++)
							if (c + q < left) out[c + q] = y[q];
					}
				}
			}
			tc_fence_before();
			__syncthreads();
			tc_fence_after();
			if (tl + 1 < tl1 && tid == 0) {
				mbar_expect_tx(&sv_bar, svbytes);
				fetch_v(tl + 1);
				fetch_s(tl + 1);
			}
		}
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(256));
}

// ------------------------------------------------------------------ norm and gate of the read-outs
// out = parts of a row normed; gate before (o silu(z)) or after (times sigmoid(z)). A warp per (row, part), V columns per
// lane at a time; the first LN_HOLD of them stay in registers between the two uses.
constexpr int LN_HOLD = 10;
template <typename OT, int V>
__global__ void __launch_bounds__(256) lin_norm_kernel(OT *out, int ldo, const float *o, int ldraw, const OT *gate, int ldg, const float *w, int R, int n, int parts,
                                                       int gate_first, float eps) {
	pdl_trigger();
	pdl_wait();
	const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
	if (i >= R * parts) return;
	const int r = i / parts, width = n / parts, c0 = (i % parts) * width;
	const float *src = o + size_t(r) * ldraw + c0;
	const OT *z = gate + size_t(r) * ldg + c0;
	float v[LN_HOLD][V], g[LN_HOLD][V];
	float q = 0.0f;
	auto take = [&](int c, float (&x)[V], float (&y)[V]) {  // y: the gate, x: what is normed
		lin_load<V>(x, src + c);
		lin_load<V>(y, z + c);
	};
	auto finish = [&](float (&x)[V], float (&y)[V]) {
#pragma unroll
		for (int e = 0; e < V; e++) {
			const float s = lin_sigmoid<OT>(y[e]);
			if (gate_first) x[e] *= y[e] * s;
			y[e] = gate_first ? 1.0f : s;
			q = fmaf(x[e], x[e], q);
		}
	};
#pragma unroll
	for (int j = 0; j < LN_HOLD; j++)
		if (V * (lane + 32 * j) < width) take(V * (lane + 32 * j), v[j], g[j]);
#pragma unroll
	for (int j = 0; j < LN_HOLD; j++)
		if (V * (lane + 32 * j) < width) finish(v[j], g[j]);
	for (int c = V * (lane + 32 * LN_HOLD); c < width; c += 32 * V) {
		float x[V], y[V];
		take(c, x, y);
		finish(x, y);
	}
	const float f = 1.0f / sqrtf(warp_sum(q) / float(width) + eps);
	OT *dst = out + size_t(r) * ldo + c0;
	auto put = [&](int c, const float (&x)[V], const float (&y)[V]) {
		float u[V];
		lin_load<V>(u, w + c0 + c);
#pragma unroll
		for (int e = 0; e < V; e++) u[e] *= x[e] * f * y[e];
		lin_store<V, OT>(dst + c, u);
	};
#pragma unroll
	for (int j = 0; j < LN_HOLD; j++)
		if (V * (lane + 32 * j) < width) put(V * (lane + 32 * j), v[j], g[j]);
	for (int c = V * (lane + 32 * LN_HOLD); c < width; c += 32 * V) {
		float x[V], y[V];
		take(c, x, y);
		finish(x, y);
		put(c, x, y);
	}
}

}  // namespace tg
