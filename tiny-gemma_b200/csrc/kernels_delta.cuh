// Gated delta rule with one decay per head and key channel. Per head, with a state S [dk][dv]:
//     S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
// q, k and v come from projections through a short causal convolution over time and silu; q and k are unit vectors
// per head (q also scaled by dk^-1/2); g_t = exp(-exp(A_log) softplus(z_t + dt_bias)). All of it in fp32.
//
// One token at a time (decoding): delta_token_cta, one CTA per (sequence, head).
//
// Portions of a prompt: the recurrence over DB = 16 tokens is solved in closed form. With D_t = g_1 .. g_t (per
// channel) and S_0 the state before the block,
//     u = T (V - Kt S_0),        Kt_t = D_t k_t,   T = (I + diag(beta) A)^-1 diag(beta),
//     o_t = (D_t q_t)^T S_0 + sum_{s<=t} M_ts u_s,   S_16 = D_16 S_0 + sum_s (D_16 / D_s) k_s u_s^T,
//     A_ts = k_t . (D_t/D_s) k_s  (s < t),   M_ts = q_t . (D_t/D_s) k_s  (s <= t),
// where every ratio D_t/D_s is formed as the product g_{s+1} .. g_t, never as a quotient, so strong decays are
// harmless. delta_block_kernel computes the block quantities (W = T Kt, D_t q_t, (D_16/D_s) k_s, T V, M) for all
// blocks and heads in parallel; delta_scan_kernel carries S through the blocks, a few columns of S per warp in
// registers; delta_out_kernel norms and gates the result.
#pragma once
#include "kernels_rowwise.cuh"
#include "tc_common.cuh"

namespace tg {

constexpr int DB = 16;  // tokens per block

struct DeltaArgs {
	StepDesc d;
	int H, KH, dk, dv, taps;
	// projections: row r at p + r * ldp; [q KH*dk][k KH*dk][v H*dv] at p_conv, beta's at p_b. Either type of element.
	const void *p;
	int ldp, p_conv, p_b;
	const float *cw;       // [taps][2*KH*dk + H*dv] convolution weights
	float *hist;           // [B][2][taps-1][2*KH*dk + H*dv] convolution inputs of earlier steps
	const float *A_log;    // [H]
	const float *dt_bias;  // [H*dk]
	const float *z;        // [R][H*dk] second decay projection     (portions)
	const float *gz;       // [R][H*dv] second gate projection      (portions)
	int ldz, ldgz;         // their row strides
	float *S;              // [B][H][dk][dv]
	const float *norm;     // [dv]
	float eps, out_scale;
	void *out;             // [R] rows of ldo; this head's dv values at column o_col + h*dv
	int ldo, o_col;
	// one token at a time: the low-rank second stages are evaluated here
	int ra, rg, p_a1, p_g1;
	const __nv_bfloat16 *a2, *g2;  // [H*dk][lda2], [H*dv][ldg2]
	int lda2, ldg2;
	// block quantities, DKP = dk rounded up to 32, 64, 128 or 256
	int dkp;
	float *blk;            // [blocks][H]: W, Q, K [DB][dkp], D [dkp], M [DB][DB] (delta_block_floats)
	float *bV;             // [blocks][H][DB][dv]: T V
	int *err;
	float *o;              // [R][H*dv] raw read-outs
};

// convolution input of channel c at time t of segment seg (t < 0: earlier steps)
template <typename PT>
__device__ __forceinline__ float delta_conv_in(const DeltaArgs &a, int row0, int pos, const float *hr, int C, int t, int c) {
	if (t >= 0) return to_f32(reinterpret_cast<const PT *>(a.p)[size_t(row0 + t) * a.ldp + a.p_conv + c]);
	return pos + t >= 0 ? hr[size_t(a.taps - 1 + t) * C + c] : 0.0f;
}
template <typename PT>
__device__ __forceinline__ float delta_conv(const DeltaArgs &a, int row0, int pos, const float *hr, int C, int t, int c) {
	float y = 0.0f;
	for (int j = 0; j < a.taps; j++) y = fmaf(a.cw[size_t(j) * C + c], delta_conv_in<PT>(a, row0, pos, hr, C, t - (a.taps - 1) + j, c), y);
	return silu_f(y);
}
// leaves the segment's last taps - 1 convolution inputs of channels [c0, c0 + n) in the other history buffer
template <typename PT>
__device__ __forceinline__ void delta_hist_save(const DeltaArgs &a, int row0, int len, int pos, const float *hr, float *hw, int C, int c0, int n) {
	for (int i = threadIdx.x; i < n * (a.taps - 1); i += blockDim.x) {
		const int q = i / n, c = c0 + i % n;
		hw[size_t(q) * C + c] = delta_conv_in<PT>(a, row0, pos, hr, C, len - (a.taps - 1) + q, c);
	}
}

// ------------------------------------------------------------------ one token
// smem: q[dk] k[dk] g[dk] v[dv] gate[dv] part[nparts*2*dv] red[64] low-rank inputs[ra + rg]. 256 threads. Row r of the step is a segment of
// length 1.
__host__ __device__ inline int delta_token_parts(int dv) { return dv >= 256 ? 1 : 256 / dv; }
// the state of a head held in registers between its two uses: 16 rows of 4 columns per thread
__host__ __device__ inline bool delta_token_in_regs(int dk, int dv) { return dk <= 128 && dv <= 128 && dv % 4 == 0; }
__host__ __device__ inline size_t delta_token_smem(int dk, int dv, int ra, int rg) {
	const int parts = delta_token_in_regs(dk, dv) ? 8 : delta_token_parts(dv);
	return (size_t(3) * dk + 2 * size_t(dv) + size_t(parts) * 2 * dv + 64 + ra + rg) * 4;
}
template <typename PT, typename OT>
__device__ void delta_token_cta(const DeltaArgs &a, int r, int h, float *sm) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int dk = a.dk, dv = a.dv, per = a.H / a.KH, kh = h / per, C = 2 * a.KH * dk + a.H * dv;
	float *sq = sm, *sk = sq + dk, *sg = sk + dk, *sv = sg + dk, *sgate = sv + dv, *part = sgate + dv;
	const bool in_regs = delta_token_in_regs(dk, dv);
	float *red = part + (in_regs ? 8 : delta_token_parts(dv)) * 2 * dv;
	const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], pos = a.d.seg_pos[seg], par = a.d.seg_par[seg];
	float *hb = a.hist + size_t(seq) * 2 * (a.taps - 1) * C;
	const float *hr = hb + size_t(par) * (a.taps - 1) * C;
	float *hw = hb + size_t(par ^ 1) * (a.taps - 1) * C;
	const PT *prow = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	// the state: with in_regs a lane owns four columns of the rows warp, warp + 8, ...; requested first
	float *S = a.S + (size_t(seq) * a.H + h) * dk * dv;
	const bool fresh = pos == 0;
	float4 st[16];
	if (in_regs) {
#pragma unroll
		for (int e = 0; e < 16; e++) {
			const int i = warp + 8 * e;
			st[e] = !fresh && i < dk && 4 * lane < dv ? *reinterpret_cast<const float4 *>(S + size_t(i) * dv + 4 * lane) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
		}
	}
	float *lr = red + 64;
	for (int i = tid; i < a.ra + a.rg; i += 256) lr[i] = to_f32(prow[i < a.ra ? a.p_a1 + i : a.p_g1 + i - a.ra]);
	// convolutions
	for (int i = tid; i < 2 * dk + dv; i += 256) {
		const int ch = i < dk ? kh * dk + i : (i < 2 * dk ? (a.KH + kh) * dk + i - dk : 2 * a.KH * dk + h * dv + i - 2 * dk);
		float y;
		if (a.taps <= 4) {  // all loads in flight together
			float w[4], x[4];
#pragma unroll
			for (int j = 0; j < 4; j++) {
				w[j] = j >= 4 - a.taps ? a.cw[size_t(j - (4 - a.taps)) * C + ch] : 0.0f;
				x[j] = j >= 4 - a.taps ? delta_conv_in<PT>(a, r, pos, hr, C, j - 3, ch) : 0.0f;
			}
			y = silu_f(fmaf(w[3], x[3], fmaf(w[2], x[2], fmaf(w[1], x[1], w[0] * x[0]))));
		} else {
			y = delta_conv<PT>(a, r, pos, hr, C, 0, ch);
		}
		(i < dk ? sq[i] : (i < 2 * dk ? sk[i - dk] : sv[i - 2 * dk])) = y;
	}
	__syncthreads();
	// low-rank second stages: eight lanes per output, 16 bytes of its row per lane and round
	{
		const float ea = expf(a.A_log[h]);
		const int sub = lane & 7;
#pragma unroll 4
		for (int o0 = 0; o0 < dk + dv; o0 += 32) {
			const int o = o0 + warp * 4 + (lane >> 3);
			const bool first = o < dk;
			const __nv_bfloat16 *w = first ? a.a2 + size_t(h * dk + o) * a.lda2 : a.g2 + size_t(h * dv + o - dk) * a.ldg2;
			const float *x = first ? lr : lr + a.ra;
			const int n = o < dk + dv ? (first ? a.ra : a.rg) : 0;
			float s = 0.0f;
#pragma unroll 2
			for (int j = 8 * sub; j < n; j += 64) {
				const uint4 u = *reinterpret_cast<const uint4 *>(w + j);
				s = fmaf(bf16_lo(u.x), x[j], s); s = fmaf(bf16_hi(u.x), x[j + 1], s);
				s = fmaf(bf16_lo(u.y), x[j + 2], s); s = fmaf(bf16_hi(u.y), x[j + 3], s);
				s = fmaf(bf16_lo(u.z), x[j + 4], s); s = fmaf(bf16_hi(u.z), x[j + 5], s);
				s = fmaf(bf16_lo(u.w), x[j + 6], s); s = fmaf(bf16_hi(u.w), x[j + 7], s);
			}
			s += __shfl_xor_sync(0xffffffffu, s, 1);
			s += __shfl_xor_sync(0xffffffffu, s, 2);
			s += __shfl_xor_sync(0xffffffffu, s, 4);
			if (sub == 0) {
				if (o < dk) sg[o] = expf(-ea * softplus_f(s + a.dt_bias[h * dk + o]));
				else if (o < dk + dv) sgate[o - dk] = sigmoid_f(s);
			}
		}
	}
	if (h % per == 0) {
		delta_hist_save<PT>(a, r, 1, pos, hr, hw, C, kh * dk, dk);
		delta_hist_save<PT>(a, r, 1, pos, hr, hw, C, (a.KH + kh) * dk, dk);
	}
	delta_hist_save<PT>(a, r, 1, pos, hr, hw, C, 2 * a.KH * dk + h * dv, dv);
	__syncthreads();
	// unit vectors
	if (warp < 2) {
		float *x = warp == 0 ? sq : sk;
		float s = 0.0f;
		for (int i = lane; i < dk; i += 32) s = fmaf(x[i], x[i], s);
		const float f = (warp == 0 ? 1.0f / sqrtf(float(dk)) : 1.0f) / sqrtf(warp_sum(s) + 1e-6f);
		for (int i = lane; i < dk; i += 32) x[i] *= f;
	}
	__syncthreads();
	if (warp == 0) {
		float s = 0.0f;
		for (int i = lane; i < dk; i += 32) s = fmaf(sq[i], sk[i], s);
		s = warp_sum(s);
		if (lane == 0) red[33] = s;
	}
	const float beta = sigmoid_f(to_f32(prow[a.p_b + h]));
	float ss = 0.0f;
	__syncthreads();
	if (in_regs) {
		float4 xk = make_float4(0.0f, 0.0f, 0.0f, 0.0f), xq = xk;
#pragma unroll
		for (int e = 0; e < 16; e++) {
			const int i = warp + 8 * e;
			if (i < dk) {
				const float gi = sg[i], ki = sk[i], qi = sq[i];
				st[e].x *= gi; st[e].y *= gi; st[e].z *= gi; st[e].w *= gi;
				xk.x = fmaf(st[e].x, ki, xk.x); xk.y = fmaf(st[e].y, ki, xk.y); xk.z = fmaf(st[e].z, ki, xk.z); xk.w = fmaf(st[e].w, ki, xk.w);
				xq.x = fmaf(st[e].x, qi, xq.x); xq.y = fmaf(st[e].y, qi, xq.y); xq.z = fmaf(st[e].z, qi, xq.z); xq.w = fmaf(st[e].w, qi, xq.w);
			}
		}
		if (4 * lane < dv) {
			float *pk = part + (warp * 2) * dv + 4 * lane, *pq = part + (warp * 2 + 1) * dv + 4 * lane;
			pk[0] = xk.x; pk[1] = xk.y; pk[2] = xk.z; pk[3] = xk.w;
			pq[0] = xq.x; pq[1] = xq.y; pq[2] = xq.z; pq[3] = xq.w;
		}
		__syncthreads();
		if (tid < dv) {  // u into sv, the read-out times the gate into sgate
			float k = 0.0f, q = 0.0f;
#pragma unroll
			for (int w = 0; w < 8; w++) {
				k += part[(w * 2) * dv + tid];
				q += part[(w * 2 + 1) * dv + tid];
			}
			const float u = beta * (sv[tid] - k), o = fmaf(u, red[33], q);
			sv[tid] = u;
			ss = o * o;
			sgate[tid] *= o;
		}
		__syncthreads();
		if (4 * lane < dv) {
			const float u0 = sv[4 * lane], u1 = sv[4 * lane + 1], u2 = sv[4 * lane + 2], u3 = sv[4 * lane + 3];
#pragma unroll
			for (int e = 0; e < 16; e++) {
				const int i = warp + 8 * e;
				if (i < dk) {
					const float ki = sk[i];
					*reinterpret_cast<float4 *>(S + size_t(i) * dv + 4 * lane) =
					    make_float4(fmaf(ki, u0, st[e].x), fmaf(ki, u1, st[e].y), fmaf(ki, u2, st[e].z), fmaf(ki, u3, st[e].w));
				}
			}
		}
	}
	// any other size: a thread owns a column (and one of `np` runs of rows) and reads it twice
	const int np = delta_token_parts(dv);
	for (int c0 = in_regs ? dv : 0; c0 < dv; c0 += 256 / np) {
		const int c = c0 + tid % (256 / np), pt = tid / (256 / np);
		const bool on = c < dv && pt < np;
		const int rows = (dk + np - 1) / np, i0 = pt * rows, i1 = min(dk, i0 + rows);
		float sk_ = 0.0f, sq_ = 0.0f;
		if (on) {
			if (!fresh) {
#pragma unroll 16
				for (int i = i0; i < i1; i++) {
					const float s = sg[i] * S[size_t(i) * dv + c];
					sk_ = fmaf(s, sk[i], sk_);
					sq_ = fmaf(s, sq[i], sq_);
				}
			}
			part[(pt * 2) * dv + c] = sk_;
			part[(pt * 2 + 1) * dv + c] = sq_;
		}
		__syncthreads();
		if (on) {
			sk_ = sq_ = 0.0f;
			for (int q = 0; q < np; q++) {
				sk_ += part[(q * 2) * dv + c];
				sq_ += part[(q * 2 + 1) * dv + c];
			}
			const float u = beta * (sv[c] - sk_);
#pragma unroll 16
			for (int i = i0; i < i1; i++) {
				float *p = S + size_t(i) * dv + c;
				*p = fmaf(sk[i], u, fresh ? 0.0f : sg[i] * *p);
			}
			const float o = fmaf(u, red[33], sq_);
			if (pt == 0) {
				ss = fmaf(o, o, ss);
				sgate[c] *= o;
			}
		}
		__syncthreads();
	}
	ss = warp_sum(ss);
	if (lane == 0) red[warp] = ss;
	__syncthreads();
	ss = 0.0f;
	for (int w = 0; w < 8; w++) ss += red[w];
	const float f = a.out_scale / sqrtf(ss / float(dv) + a.eps);
	for (int c = tid; c < dv; c += 256)
		reinterpret_cast<OT *>(a.out)[size_t(r) * a.ldo + a.o_col + h * dv + c] = from_f32<OT>(sgate[c] * f * a.norm[c]);
}

// ------------------------------------------------------------------ blocks of a portion
__host__ __device__ inline int delta_block_base(int seg_row, int seg) { return seg_row / DB + seg; }

__host__ __device__ constexpr size_t delta_block_floats(int dkp) { return size_t(3) * DB * dkp + dkp + DB * DB; }

// smem floats: k, q, g, p [DB][dkp], v [DB][dv], A, M, T [DB][DB], beta [DB]
__host__ __device__ inline size_t delta_block_smem(int dkp, int dv) { return (size_t(3) * DB * dkp + size_t(DB) * dv + 3 * DB * DB + DB) * 4; }

// grid (blocks of the longest segment, H, segments), 256 threads
template <typename PT>
__global__ void __launch_bounds__(256, 3) delta_block_kernel(DeltaArgs a) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ __align__(16) float db_sm[];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int blk = blockIdx.x, h = blockIdx.y, seg = blockIdx.z;
	const int len = a.d.seg_len[seg], t0 = blk * DB;
	if (t0 >= len) return;
	const int n = min(DB, len - t0);
	const int row0 = a.d.seg_row[seg], pos = a.d.seg_pos[seg], seq = a.d.seg_seq[seg], par = a.d.seg_par[seg];
	const int dk = a.dk, dv = a.dv, dkp = a.dkp, per = a.H / a.KH, kh = h / per, C = 2 * a.KH * dk + a.H * dv;
	float *hb = a.hist + size_t(seq) * 2 * (a.taps - 1) * C;
	const float *hr = hb + size_t(par) * (a.taps - 1) * C;
	float *hw = hb + size_t(par ^ 1) * (a.taps - 1) * C;
	float *sk = db_sm, *sq = sk + DB * dkp, *sg = sq + DB * dkp, *sv = sg + DB * dkp, *sA = sv + DB * dv, *sM = sA + DB * DB, *sT = sM + DB * DB,
	      *sb = sT + DB * DB;
	// q, k, g, v, beta; tokens past the end change nothing (g = 1, everything else 0)
	const float ea = expf(a.A_log[h]);
	constexpr int HB = DB / 2;  // a thread walks a channel down half of the block's tokens
	for (int i = tid; i < 2 * (2 * dkp + dv); i += 256) {
		const int part = i >= 2 * dkp + dv, f = part * HB, e = i - part * (2 * dkp + dv);
		const int kind = e < dkp ? 0 : (e < 2 * dkp ? 1 : 2), c = kind == 0 ? e : (kind == 1 ? e - dkp : e - 2 * dkp);
		const int ld = kind == 2 ? dv : dkp;
		float *dst = (kind == 0 ? sq : (kind == 1 ? sk : sv)) + f * ld + c;
		if (kind < 2 && c >= dk) {
			for (int t = 0; t < HB; t++) dst[t * ld] = 0.0f;
			continue;
		}
		const int ch = kind == 0 ? kh * dk + c : (kind == 1 ? (a.KH + kh) * dk + c : 2 * a.KH * dk + h * dv + c);
		if (a.taps <= 4) {
			float x[HB + 3], w[4];
#pragma unroll
			for (int j = 0; j < 4; j++) w[j] = j >= 4 - a.taps ? a.cw[size_t(j - (4 - a.taps)) * C + ch] : 0.0f;
			const int tf = t0 + f - 3;
			if (tf >= 0) {  // no history: plain rows (those past the segment's end are not used)
				const PT *px = reinterpret_cast<const PT *>(a.p) + size_t(row0 + tf) * a.ldp + a.p_conv + ch;
#pragma unroll
				for (int j = 0; j < HB + 3; j++) x[j] = f + j - 3 < n ? to_f32(px[size_t(j) * a.ldp]) : 0.0f;
			} else {
#pragma unroll
				for (int j = 0; j < HB + 3; j++) x[j] = f + j - 3 < n && 3 - j < a.taps ? delta_conv_in<PT>(a, row0, pos, hr, C, tf + j, ch) : 0.0f;
			}
#pragma unroll
			for (int t = 0; t < HB; t++) {
				const float y = fmaf(w[3], x[t + 3], fmaf(w[2], x[t + 2], fmaf(w[1], x[t + 1], w[0] * x[t])));
				dst[t * ld] = f + t < n ? __fdividef(y, 1.0f + __expf(-y)) : 0.0f;
			}
		} else {
			for (int t = 0; t < HB; t++) dst[t * ld] = f + t < n ? delta_conv<PT>(a, row0, pos, hr, C, t0 + f + t, ch) : 0.0f;
		}
	}
	for (int i = tid; i < 2 * dkp; i += 256) {
		const int part = i >= dkp, f = part * HB, c = i - part * dkp;
		const float bias = c < dk ? a.dt_bias[h * dk + c] : 0.0f;
		float zv[HB];
#pragma unroll
		for (int t = 0; t < HB; t++) zv[t] = f + t < n && c < dk ? a.z[size_t(row0 + t0 + f + t) * a.ldz + h * dk + c] : 0.0f;
#pragma unroll
		for (int t = 0; t < HB; t++) sg[(f + t) * dkp + c] = f + t < n && c < dk ? expf(-ea * softplus_f(zv[t] + bias)) : 1.0f;
	}
	if (tid < DB) sb[tid] = tid < n ? sigmoid_f(to_f32(reinterpret_cast<const PT *>(a.p)[size_t(row0 + t0 + tid) * a.ldp + a.p_b + h])) : 0.0f;
	if (t0 + DB >= len) {  // the segment's last block
		if (h % per == 0) {
			delta_hist_save<PT>(a, row0, len, pos, hr, hw, C, kh * dk, dk);
			delta_hist_save<PT>(a, row0, len, pos, hr, hw, C, (a.KH + kh) * dk, dk);
		}
		delta_hist_save<PT>(a, row0, len, pos, hr, hw, C, 2 * a.KH * dk + h * dv, dv);
	}
	__syncthreads();
	// unit vectors: a warp per token
	for (int t = warp; t < DB; t += 8) {
		float nk = 0.0f, nq = 0.0f;
		for (int c = lane; c < dkp; c += 32) {
			nk = fmaf(sk[t * dkp + c], sk[t * dkp + c], nk);
			nq = fmaf(sq[t * dkp + c], sq[t * dkp + c], nq);
		}
		const float fk = 1.0f / sqrtf(warp_sum(nk) + 1e-6f), fq = 1.0f / (sqrtf(float(dk)) * sqrtf(warp_sum(nq) + 1e-6f));
		for (int c = lane; c < dkp; c += 32) {
			sk[t * dkp + c] *= fk;
			sq[t * dkp + c] *= fq;
		}
	}
	__syncthreads();
	// A and M, columns s1 = warp and s2 = 15 - warp: p = k_s decayed step by step. A lane takes the channels lane,
	// lane + 32, ...; the four sums of a step are reduced together.
	{
		const int s1 = warp, s2 = DB - 1 - warp;
		float p1[8], p2[8];
#pragma unroll
		for (int j = 0; j < 8; j++) {
			p1[j] = lane + 32 * j < dkp ? sk[s1 * dkp + lane + 32 * j] : 0.0f;
			p2[j] = lane + 32 * j < dkp ? sk[s2 * dkp + lane + 32 * j] : 0.0f;
		}
		for (int t = 0; t < DB; t++) {
			float xa = 0.0f, xm = 0.0f, ya = 0.0f, ym = 0.0f;  // columns s1 (x) and s2 (y) of A and M
			if (t >= s1) {
#pragma unroll
				for (int j = 0; j < 8; j++)
					if (32 * j < dkp) {
						const int i = t * dkp + lane + 32 * j;
						const float k = sk[i], q = sq[i], g = sg[i];
						if (t > s1) p1[j] *= g;
						xa = fmaf(k, p1[j], xa);
						xm = fmaf(q, p1[j], xm);
						if (t >= s2) {
							if (t > s2) p2[j] *= g;
							ya = fmaf(k, p2[j], ya);
							ym = fmaf(q, p2[j], ym);
						}
					}
				const bool hi = lane & 16, mid = lane & 8;
				const float a1 = (hi ? ya : xa) + __shfl_xor_sync(0xffffffffu, hi ? xa : ya, 16), m1 = (hi ? ym : xm) + __shfl_xor_sync(0xffffffffu, hi ? xm : ym, 16);
				float v = (mid ? m1 : a1) + __shfl_xor_sync(0xffffffffu, mid ? a1 : m1, 8);
				v += __shfl_xor_sync(0xffffffffu, v, 4);
				v += __shfl_xor_sync(0xffffffffu, v, 2);
				v += __shfl_xor_sync(0xffffffffu, v, 1);
				xa = v;  // lanes 0, 8, 16, 24: A s1, M s1, A s2, M s2
			}
			if ((lane & 7) == 0) {
				const int s = lane & 16 ? s2 : s1;
				const bool isM = lane & 8;
				(isM ? sM : sA)[t * DB + s] = (isM ? t >= s : t > s) ? xa : 0.0f;
			}
		}
	}
	__syncthreads();
	const size_t bh = (size_t(delta_block_base(row0, seg)) + blk) * a.H + h;
	if (tid < DB) {  // column tid of T by forward substitution
		float x[DB];
#pragma unroll
		for (int t = 0; t < DB; t++) {
			float s = t == tid ? 1.0f : 0.0f;
#pragma unroll
			for (int j = 0; j < t; j++) s = fmaf(-sA[t * DB + j], x[j], s);
			x[t] = sb[t] * s;
			sT[t * DB + tid] = x[t];
		}
	}
	float *gW = a.blk + bh * delta_block_floats(dkp), *gQ = gW + DB * dkp, *gK = gQ + DB * dkp, *gD = gK + DB * dkp, *gM = gD + dkp;
	if (tid >= 64 && tid < 64 + DB * DB / 4) reinterpret_cast<float4 *>(gM)[tid - 64] = reinterpret_cast<float4 *>(sM)[tid - 64];
	// per channel: D_t k_t, D_t q_t, and the suffix products
	for (int c = tid; c < dkp; c += 256) {
		float D = 1.0f, suf[DB];
		suf[DB - 1] = 1.0f;
#pragma unroll
		for (int t = DB - 1; t > 0; t--) suf[t - 1] = suf[t] * sg[t * dkp + c];
#pragma unroll
		for (int t = 0; t < DB; t++) {
			const float k = sk[t * dkp + c];
			D *= sg[t * dkp + c];
			gK[t * dkp + c] = suf[t] * k;
			gQ[t * dkp + c] = D * sq[t * dkp + c];
			sk[t * dkp + c] = D * k;
		}
		gD[c] = D;
	}
	__syncthreads();
	// W = T Kt and T V
	for (int c = tid; c < dkp + dv; c += 256) {
		const float *src = c < dkp ? sk + c : sv + (c - dkp);
		const int ld = c < dkp ? dkp : dv;
		float *dst = c < dkp ? gW + c : a.bV + bh * DB * dv + (c - dkp);
		float x[DB];
#pragma unroll
		for (int t = 0; t < DB; t++) x[t] = src[t * ld];
#pragma unroll
		for (int t = 0; t < DB; t++) {
			float s = 0.0f;  // (T is zero above the diagonal)
#pragma unroll
			for (int j = 0; j <= t; j += 4) {
				const float4 w = *reinterpret_cast<const float4 *>(sT + t * DB + j);
				s = fmaf(w.x, x[j], fmaf(w.y, x[j + 1], fmaf(w.z, x[j + 2], fmaf(w.w, x[j + 3], s))));
			}
			dst[size_t(t) * ld] = s;
		}
	}
}

// ------------------------------------------------------------------ carrying the state through the blocks
// grid (column groups of 4 NC, H, segments), NW warps. The CTA holds 4 NC columns of S in registers: warp w rows
// 8 RPL w .. , a lane RPL of them (4 (lane & 7) + 32 j + {0..3}) of columns 4 NC x + (lane >> 3) + 4 i. The chain over
// the blocks is sequential and a block is a few hundred instructions per warp, so what counts is its latency: the block
// quantities of a (block, head) are one bulk copy, `stages` of them in flight; rows are read from shared memory a group
// ahead of their use; the products run on packed fp32 pairs; and the warps meet at one barrier per block.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
	float2 d;
	asm("fma.rn.f32x2 %0, %1, %2, %3;"
	    : "=l"(reinterpret_cast<unsigned long long &>(d))
	    : "l"(reinterpret_cast<const unsigned long long &>(a)), "l"(reinterpret_cast<const unsigned long long &>(b)), "l"(reinterpret_cast<const unsigned long long &>(c)));
	return d;
}
// (volatile: the loads stay where they are written, ahead of their use)
__device__ __forceinline__ float4 ds_ld4(const float *p) {
	float4 v;
	asm volatile("ld.shared.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(smem_u32(p)) : "memory");
	return v;
}
// acc[16] per lane -> the sums over the 8 lanes of a column for tokens 2 rl, 2 rl + 1
__device__ __forceinline__ float2 delta_reduce(const float (&acc)[DB], int rl) {
	float r1[8], r2[4];
	const bool h4 = rl & 4, h2 = rl & 2, h1 = rl & 1;
#pragma unroll
	for (int i = 0; i < 8; i++) r1[i] = (h4 ? acc[8 + i] : acc[i]) + __shfl_xor_sync(0xffffffffu, h4 ? acc[i] : acc[8 + i], 4);
#pragma unroll
	for (int i = 0; i < 4; i++) r2[i] = (h2 ? r1[4 + i] : r1[i]) + __shfl_xor_sync(0xffffffffu, h2 ? r1[i] : r1[4 + i], 2);
	float2 o;
	o.x = (h1 ? r2[2] : r2[0]) + __shfl_xor_sync(0xffffffffu, h1 ? r2[0] : r2[2], 1);
	o.y = (h1 ? r2[3] : r2[1]) + __shfl_xor_sync(0xffffffffu, h1 ? r2[1] : r2[3], 1);
	return o;
}
constexpr int DS_MAX_STAGES = 4;
template <int RPL, int NW, int NC> size_t delta_scan_smem(int stages) {
	return (size_t(stages) * delta_block_floats(8 * RPL * NW) + size_t(5) * NW * 4 * NC * 20) * 4;
}

template <int RPL, int NW, int NC>
__global__ void __launch_bounds__(32 * NW) delta_scan_kernel(DeltaArgs a, int stages) {
	pdl_trigger();
	constexpr int DKP = 8 * RPL * NW, COLS = 4 * NC;
	constexpr size_t BF = delta_block_floats(DKP);
	extern __shared__ __align__(128) float ds_sm[];
	__shared__ uint64_t full_bar[DS_MAX_STAGES];
	__shared__ int s_fail;
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int h = blockIdx.y, seg = blockIdx.z, rl = lane & 7, cl = lane >> 3;
	float *pw = ds_sm + size_t(stages) * BF;          // [2][NW][COLS][20] partial W dots
	float *pq = pw + 2 * NW * COLS * 20;              // the same of Q
	float *su = pq + 2 * NW * COLS * 20 + warp * COLS * 20;  // this warp's copy of u [COLS][20]
	if (tid == 0) {
		for (int i = 0; i < stages; i++) mbar_init(&full_bar[i], 1);
		s_fail = 0;
		asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
	}
	__syncthreads();
	pdl_wait();
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], pos = a.d.seg_pos[seg], seq = a.d.seg_seq[seg];
	const int nb = (len + DB - 1) / DB, dk = a.dk, dv = a.dv;
	const size_t blk0 = delta_block_base(row0, seg);
	auto fetch = [&](int b) {
		if (tid == 0) {
			fence_proxy_async();
			mbar_expect_tx(&full_bar[b % stages], uint32_t(BF * 4));
			asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(ds_sm + size_t(b % stages) * BF)),
			             "l"(a.blk + ((blk0 + b) * a.H + h) * BF), "r"(uint32_t(BF * 4)), "r"(smem_u32(&full_bar[b % stages]))
			             : "memory");
		}
	};
	int issued = min(stages - 1, nb);
	for (int b = 0; b < issued; b++) fetch(b);
	int col[NC];
	float2 S[NC][RPL / 2];
	float *Sg = a.S + (size_t(seq) * a.H + h) * dk * dv;
	const int r_base = warp * 8 * RPL + 4 * rl;
#pragma unroll
	for (int x = 0; x < NC; x++) {
		col[x] = (blockIdx.x * NC + x) * 4 + cl;
#pragma unroll
		for (int j = 0; j < RPL / 2; j++) {
			const int i = r_base + 32 * (j >> 1) + 2 * (j & 1);
			S[x][j].x = (pos > 0 && col[x] < dv && i < dk) ? Sg[size_t(i) * dv + col[x]] : 0.0f;
			S[x][j].y = (pos > 0 && col[x] < dv && i + 1 < dk) ? Sg[size_t(i + 1) * dv + col[x]] : 0.0f;
		}
	}
	float2 v[NC];
	auto load_v = [&](int b) {
		const float *vb = a.bV + ((blk0 + b) * a.H + h) * DB * dv + size_t(2 * rl) * dv;
#pragma unroll
		for (int x = 0; x < NC; x++) v[x] = col[x] < dv ? make_float2(vb[col[x]], vb[dv + col[x]]) : make_float2(0.0f, 0.0f);
	};
	load_v(0);
	for (int b = 0; b < nb; b++) {
		const int par = b & 1;
		if (!tc_wait(&full_bar[b % stages], (b / stages) & 1, a.err)) s_fail = 1;
		const float *sW = ds_sm + size_t(b % stages) * BF, *sD = sW + 3 * DB * DKP, *sM = sD + DKP;
		// W, Q and K are read as one stream of groups of TG token rows, a group ahead of its use
		constexpr int TG = RPL >= 8 ? 4 : 8, GR = DB / TG;
		float4 cur[TG][RPL / 4], nxt[TG][RPL / 4];
		auto rows = [&](int g, float4 (&w)[TG][RPL / 4]) {  // g: 0 .. 3 GR - 1 (W, Q and K lie one after the other)
#pragma unroll
			for (int t = 0; t < TG; t++)
#pragma unroll
				for (int j = 0; j < RPL / 4; j++) w[t][j] = ds_ld4(sW + (g * TG + t) * DKP + r_base + 32 * j);
		};
		float acc[NC][DB];
		auto dots = [&](int g) {
#pragma unroll
			for (int t = 0; t < TG; t++)
#pragma unroll
				for (int x = 0; x < NC; x++) {
					float2 s = make_float2(0.0f, 0.0f);
#pragma unroll
					for (int j = 0; j < RPL / 4; j++) {
						s = fma2(make_float2(cur[t][j].x, cur[t][j].y), S[x][2 * j], s);
						s = fma2(make_float2(cur[t][j].z, cur[t][j].w), S[x][2 * j + 1], s);
					}
					acc[x][(g % GR) * TG + t] = s.x + s.y;
				}
		};
		auto shift = [&] {
#pragma unroll
			for (int t = 0; t < TG; t++)
#pragma unroll
				for (int j = 0; j < RPL / 4; j++) cur[t][j] = nxt[t][j];
		};
		rows(0, cur);
#pragma unroll
		for (int g = 0; g < 2 * GR; g++) {
			rows(g + 1, nxt);
			dots(g);
			shift();
			if (g == GR - 1 || g == 2 * GR - 1) {
				float *dst = (g == GR - 1 ? pw : pq) + (par * NW + warp) * COLS * 20;
#pragma unroll
				for (int x = 0; x < NC; x++) *reinterpret_cast<float2 *>(dst + (4 * x + cl) * 20 + 2 * rl) = delta_reduce(acc[x], rl);
			}
		}
		if (NW > 1) __syncthreads();
		else __syncwarp();
		if (*(volatile int *)&s_fail) {
			for (int q = b + 1; q < issued; q++) tc_wait(&full_bar[q % stages], (q / stages) & 1, a.err);  // copies in flight land first
			break;
		}
		if (issued < nb) fetch(issued++);  // (every warp is past the block that used this stage)
#pragma unroll
		for (int x = 0; x < NC; x++) {
			float2 u = v[x];
#pragma unroll
			for (int w = 0; w < NW; w++) {
				const float2 d = *reinterpret_cast<const float2 *>(pw + ((par * NW + w) * COLS + 4 * x + cl) * 20 + 2 * rl);
				u.x -= d.x;
				u.y -= d.y;
			}
			*reinterpret_cast<float2 *>(su + (4 * x + cl) * 20 + 2 * rl) = u;
		}
		if (b + 1 < nb) load_v(b + 1);
		__syncwarp();
#pragma unroll
		for (int j = 0; j < RPL / 4; j++) {
			const float4 g = *reinterpret_cast<const float4 *>(sD + r_base + 32 * j);
#pragma unroll
			for (int x = 0; x < NC; x++) {
				S[x][2 * j].x *= g.x; S[x][2 * j].y *= g.y;
				S[x][2 * j + 1].x *= g.z; S[x][2 * j + 1].y *= g.w;
			}
		}
#pragma unroll
		for (int g = 2 * GR; g < 3 * GR; g++) {
			if (g + 1 < 3 * GR) rows(g + 1, nxt);
#pragma unroll
			for (int x = 0; x < NC; x++) {
				float u[TG];
#pragma unroll
				for (int t = 0; t < TG; t += 4) *reinterpret_cast<float4 *>(&u[t]) = *reinterpret_cast<const float4 *>(su + (4 * x + cl) * 20 + (g - 2 * GR) * TG + t);
#pragma unroll
				for (int t = 0; t < TG; t++)
#pragma unroll
					for (int j = 0; j < RPL / 4; j++) {
						S[x][2 * j] = fma2(make_float2(cur[t][j].x, cur[t][j].y), make_float2(u[t], u[t]), S[x][2 * j]);
						S[x][2 * j + 1] = fma2(make_float2(cur[t][j].z, cur[t][j].w), make_float2(u[t], u[t]), S[x][2 * j + 1]);
					}
			}
			if (g + 1 < 3 * GR) shift();
		}
		// read-outs: the warps share the 16 tokens; two lanes per (token, column), each half of the sum over s
#pragma unroll
		for (int e = 0; e < 4 * NC / NW + (4 * NC % NW != 0); e++) {
			const int item = (e * NW + warp) * 16 + (lane >> 1), half = lane & 1;  // 16 items per warp and round
			const int t = item / COLS, c = item % COLS;
			if (item < DB * COLS) {
				float o = 0.0f;
#pragma unroll
				for (int i = 0; i < 2; i++) {  // (M is zero above the diagonal)
					const float4 m = *reinterpret_cast<const float4 *>(sM + t * DB + 8 * half + 4 * i), u = *reinterpret_cast<const float4 *>(su + c * 20 + 8 * half + 4 * i);
					o = fmaf(m.x, u.x, o); o = fmaf(m.y, u.y, o); o = fmaf(m.z, u.z, o); o = fmaf(m.w, u.w, o);
				}
#pragma unroll
				for (int w = 0; w < NW; w++)
					if ((w & 1) == half || NW == 1) o += NW == 1 && half ? 0.0f : pq[((par * NW + w) * COLS + c) * 20 + t];
				o += __shfl_xor_sync(0xffffffffu, o, 1);
				const int gc = blockIdx.x * COLS + c;
				if (half == 0 && gc < dv && b * DB + t < len) a.o[size_t(row0 + b * DB + t) * a.H * dv + h * dv + gc] = o;
			}
		}
	}
#pragma unroll
	for (int x = 0; x < NC; x++)
#pragma unroll
		for (int j = 0; j < RPL / 2; j++) {
			const int i = r_base + 32 * (j >> 1) + 2 * (j & 1);
			if (col[x] < dv && i < dk) Sg[size_t(i) * dv + col[x]] = S[x][j].x;
			if (col[x] < dv && i + 1 < dk) Sg[size_t(i + 1) * dv + col[x]] = S[x][j].y;
		}
}

// out = rms_norm(o) * norm * sigmoid(gz) * out_scale: a warp per (row, head)
template <typename OT>
__global__ void __launch_bounds__(256) delta_out_kernel(DeltaArgs a, int R) {
	pdl_trigger();
	pdl_wait();
	const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
	if (i >= R * a.H) return;
	const int r = i / a.H, h = i % a.H, dv = a.dv;
	const float *o = a.o + size_t(r) * a.H * dv + h * dv, *gz = a.gz + size_t(r) * a.ldgz + h * dv;
	float ss = 0.0f;
	for (int c = lane; c < dv; c += 32) ss = fmaf(o[c], o[c], ss);
	const float f = a.out_scale / sqrtf(warp_sum(ss) / float(dv) + a.eps);
	OT *out = reinterpret_cast<OT *>(a.out) + size_t(r) * a.ldo + a.o_col + h * dv;
	for (int c = lane; c < dv; c += 32) out[c] = from_f32<OT>(o[c] * f * a.norm[c] * sigmoid_f(gz[c]));
}

}  // namespace tg
