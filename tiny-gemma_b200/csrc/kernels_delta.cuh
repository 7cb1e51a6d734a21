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
	float *bW, *bQ, *bK;   // [blocks][H][DB][dkp]
	float *bD;             // [blocks][H][dkp]
	float *bV;             // [blocks][H][DB][dv]
	float *bM;             // [blocks][H][DB][DB]
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
// smem: q[dk] k[dk] g[dk] v[dv] gate[dv] part[nparts*2*dv] red[32]. 256 threads. Row r of the step is a segment of
// length 1.
__host__ __device__ inline int delta_token_parts(int dv) { return dv >= 256 ? 1 : 256 / dv; }
__host__ __device__ inline size_t delta_token_smem(int dk, int dv) {
	return (size_t(3) * dk + 2 * size_t(dv) + size_t(delta_token_parts(dv)) * 2 * dv + 64) * 4;
}
template <typename PT, typename OT>
__device__ void delta_token_cta(const DeltaArgs &a, int r, int h, float *sm) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int dk = a.dk, dv = a.dv, per = a.H / a.KH, kh = h / per, C = 2 * a.KH * dk + a.H * dv;
	float *sq = sm, *sk = sq + dk, *sg = sk + dk, *sv = sg + dk, *sgate = sv + dv, *part = sgate + dv;
	float *red = part + delta_token_parts(dv) * 2 * dv;
	const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], pos = a.d.seg_pos[seg], par = a.d.seg_par[seg];
	float *hb = a.hist + size_t(seq) * 2 * (a.taps - 1) * C;
	const float *hr = hb + size_t(par) * (a.taps - 1) * C;
	float *hw = hb + size_t(par ^ 1) * (a.taps - 1) * C;
	const PT *prow = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	// convolutions
	for (int i = tid; i < 2 * dk + dv; i += 256) {
		if (i < dk) sq[i] = delta_conv<PT>(a, r, pos, hr, C, 0, kh * dk + i);
		else if (i < 2 * dk) sk[i - dk] = delta_conv<PT>(a, r, pos, hr, C, 0, (a.KH + kh) * dk + i - dk);
		else sv[i - 2 * dk] = delta_conv<PT>(a, r, pos, hr, C, 0, 2 * a.KH * dk + h * dv + i - 2 * dk);
	}
	// low-rank second stages: eight lanes per output
	{
		const float ea = expf(a.A_log[h]);
		const int sub = lane & 7;
		for (int o0 = 0; o0 < dk + dv; o0 += 32) {
			const int o = o0 + warp * 4 + (lane >> 3);
			float s = 0.0f;
			if (o < dk) {
				const __nv_bfloat16 *w = a.a2 + size_t(h * dk + o) * a.lda2;
				for (int j = sub; j < a.ra; j += 8) s = fmaf(__bfloat162float(w[j]), to_f32(prow[a.p_a1 + j]), s);
			} else if (o < dk + dv) {
				const __nv_bfloat16 *w = a.g2 + size_t(h * dv + o - dk) * a.ldg2;
				for (int j = sub; j < a.rg; j += 8) s = fmaf(__bfloat162float(w[j]), to_f32(prow[a.p_g1 + j]), s);
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
	// the state: a thread owns a column (and one of `np` runs of rows)
	float *S = a.S + (size_t(seq) * a.H + h) * dk * dv;
	const int np = delta_token_parts(dv);
	const bool fresh = pos == 0;
	float ss = 0.0f;
	__syncthreads();
	for (int c0 = 0; c0 < dv; c0 += 256 / np) {
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

// smem floats: k, q, g, p [DB][dkp], v [DB][dv], A, M, T [DB][DB], beta [DB]
__host__ __device__ inline size_t delta_block_smem(int dkp, int dv) { return (size_t(3) * DB * dkp + size_t(DB) * dv + 3 * DB * DB + DB) * 4; }

// grid (blocks of the longest segment, H, segments), 256 threads
template <typename PT>
__global__ void __launch_bounds__(256) delta_block_kernel(DeltaArgs a) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ float db_sm[];
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
	for (int i = tid; i < DB * dkp; i += 256) {
		const int t = i / dkp, c = i % dkp;
		float k = 0.0f, q = 0.0f, g = 1.0f;
		if (t < n && c < dk) {
			q = delta_conv<PT>(a, row0, pos, hr, C, t0 + t, kh * dk + c);
			k = delta_conv<PT>(a, row0, pos, hr, C, t0 + t, (a.KH + kh) * dk + c);
			g = expf(-ea * softplus_f(a.z[size_t(row0 + t0 + t) * a.ldz + h * dk + c] + a.dt_bias[h * dk + c]));
		}
		sk[i] = k;
		sq[i] = q;
		sg[i] = g;
	}
	for (int i = tid; i < DB * dv; i += 256) {
		const int t = i / dv, c = i % dv;
		sv[i] = t < n ? delta_conv<PT>(a, row0, pos, hr, C, t0 + t, 2 * a.KH * dk + h * dv + c) : 0.0f;
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
	// A and M, column s: p = k_s decayed step by step. A warp takes the columns s = warp and 15 - warp (17 steps in
	// all for every warp), a lane the channels lane, lane + 32, ...
	for (int half = 0; half < 2; half++) {
		const int s = half ? DB - 1 - warp : warp;
		float p[8];
#pragma unroll
		for (int j = 0; j < 8; j++) p[j] = lane + 32 * j < dkp ? sk[s * dkp + lane + 32 * j] : 0.0f;
		for (int t = 0; t < s; t++)
			if (lane == 0) sA[t * DB + s] = sM[t * DB + s] = 0.0f;
		for (int t = s; t < DB; t++) {
			float xa = 0.0f, xm = 0.0f;
#pragma unroll
			for (int j = 0; j < 8; j++)
				if (lane + 32 * j < dkp) {
					const int i = t * dkp + lane + 32 * j;
					if (t > s) p[j] *= sg[i];
					xa = fmaf(sk[i], p[j], xa);
					xm = fmaf(sq[i], p[j], xm);
				}
			xa = warp_sum(xa);
			xm = warp_sum(xm);
			if (lane == 0) {
				sA[t * DB + s] = t > s ? xa : 0.0f;
				sM[t * DB + s] = xm;
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
	if (tid >= 64 && tid < 64 + DB * DB / 4) reinterpret_cast<float4 *>(a.bM + bh * DB * DB)[tid - 64] = reinterpret_cast<float4 *>(sM)[tid - 64];
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
			a.bK[(bh * DB + t) * dkp + c] = suf[t] * k;
			a.bQ[(bh * DB + t) * dkp + c] = D * sq[t * dkp + c];
			sk[t * dkp + c] = D * k;
		}
		a.bD[bh * dkp + c] = D;
	}
	__syncthreads();
	// W = T Kt and T V
	for (int c = tid; c < dkp + dv; c += 256) {
		const float *src = c < dkp ? sk + c : sv + (c - dkp);
		const int ld = c < dkp ? dkp : dv;
		float *dst = c < dkp ? a.bW + bh * DB * dkp + c : a.bV + bh * DB * dv + (c - dkp);
		float x[DB];
#pragma unroll
		for (int t = 0; t < DB; t++) x[t] = src[t * ld];
#pragma unroll
		for (int t = 0; t < DB; t++) {
			float s = 0.0f;
#pragma unroll
			for (int j = 0; j <= t; j++) s = fmaf(sT[t * DB + j], x[j], s);
			dst[size_t(t) * ld] = s;
		}
	}
}

// ------------------------------------------------------------------ carrying the state through the blocks
// grid (column groups of 16, H, segments), 128 threads = 4 warps of 4 columns. A lane holds RPL rows of one column:
// rows 4 (lane & 7) + 32 j + {0..3}; the eight lanes of a column meet by butterflies.
template <int RPL>
__global__ void __launch_bounds__(128) delta_scan_kernel(DeltaArgs a) {
	pdl_trigger();
	pdl_wait();
	constexpr int DKP = 8 * RPL;
	constexpr int STAGE = 3 * DB * DKP + DKP + DB * DB + DB * 16;  // W, Q, K, D, M, V columns
	extern __shared__ __align__(16) float ds_sm[];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int h = blockIdx.y, seg = blockIdx.z, c0 = blockIdx.x * 16;
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], pos = a.d.seg_pos[seg], seq = a.d.seg_seq[seg];
	const int nb = (len + DB - 1) / DB, dk = a.dk, dv = a.dv;
	const int rl = lane & 7, c = c0 + warp * 4 + (lane >> 3);
	const bool on = c < dv;
	const size_t blk0 = delta_block_base(row0, seg);
	float S[RPL];
	float *Sg = a.S + (size_t(seq) * a.H + h) * dk * dv;
#pragma unroll
	for (int j = 0; j < RPL; j++) {
		const int i = 4 * rl + 32 * (j >> 2) + (j & 3);
		S[j] = (on && pos > 0 && i < dk) ? Sg[size_t(i) * dv + c] : 0.0f;
	}
	auto fetch = [&](int b) {
		float *st = ds_sm + (b & 1) * STAGE;
		const size_t bh = (blk0 + b) * a.H + h;
		auto cp = [&](float *dst, const float *src, int n4) {
			for (int i = tid; i < n4; i += 128)
				asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(uint32_t(__cvta_generic_to_shared(dst + 4 * i))), "l"(src + 4 * i) : "memory");
		};
		cp(st, a.bW + bh * DB * DKP, DB * DKP / 4);
		cp(st + DB * DKP, a.bQ + bh * DB * DKP, DB * DKP / 4);
		cp(st + 2 * DB * DKP, a.bK + bh * DB * DKP, DB * DKP / 4);
		cp(st + 3 * DB * DKP, a.bD + bh * DKP, DKP / 4);
		cp(st + 3 * DB * DKP + DKP, a.bM + bh * DB * DB, DB * DB / 4);
		float *v = st + 3 * DB * DKP + DKP + DB * DB;
		for (int i = tid; i < DB * 16; i += 128) {
			const int t = i >> 4, cc = c0 + (i & 15);
			if (cc < dv)
				asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(uint32_t(__cvta_generic_to_shared(v + i))), "l"(a.bV + (bh * DB + t) * dv + cc) : "memory");
			else
				v[i] = 0.0f;
		}
		asm volatile("cp.async.commit_group;" ::: "memory");
	};
	fetch(0);
	for (int b = 0; b < nb; b++) {
		if (b + 1 < nb) {
			fetch(b + 1);
			asm volatile("cp.async.wait_group 1;" ::: "memory");
		} else {
			asm volatile("cp.async.wait_group 0;" ::: "memory");
		}
		__syncthreads();
		const float *st = ds_sm + (b & 1) * STAGE;
		const float *sW = st, *sQ = st + DB * DKP, *sK = st + 2 * DB * DKP, *sD = st + 3 * DB * DKP, *sM = sD + DKP, *sV = sM + DB * DB;
		// dots of every token's W and Q with this column of S: acc[t] = W_t . S, acc[16 + t] = Q_t . S
		float acc[2 * DB];
#pragma unroll
		for (int t = 0; t < DB; t++) {
			float x = 0.0f, y = 0.0f;
#pragma unroll
			for (int j = 0; j < RPL / 4; j++) {
				const float4 w = *reinterpret_cast<const float4 *>(sW + t * DKP + 4 * rl + 32 * j);
				const float4 q = *reinterpret_cast<const float4 *>(sQ + t * DKP + 4 * rl + 32 * j);
				x = fmaf(w.x, S[4 * j], x); x = fmaf(w.y, S[4 * j + 1], x); x = fmaf(w.z, S[4 * j + 2], x); x = fmaf(w.w, S[4 * j + 3], x);
				y = fmaf(q.x, S[4 * j], y); y = fmaf(q.y, S[4 * j + 1], y); y = fmaf(q.z, S[4 * j + 2], y); y = fmaf(q.w, S[4 * j + 3], y);
			}
			acc[t] = x;
			acc[DB + t] = y;
		}
		// reduce over the 8 lanes of the column; lane rl ends with tokens 2 rl, 2 rl + 1 of both
		float w2[2], q2[2];
		{
			float r1[DB];
			const bool hi4 = rl & 4;
#pragma unroll
			for (int i = 0; i < 8; i++) {  // tokens (hi4 ? 8 + i : i)
				const float sw = hi4 ? acc[i] : acc[8 + i], kw = hi4 ? acc[8 + i] : acc[i];
				const float sq = hi4 ? acc[DB + i] : acc[DB + 8 + i], kq = hi4 ? acc[DB + 8 + i] : acc[DB + i];
				r1[i] = kw + __shfl_xor_sync(0xffffffffu, sw, 4);
				r1[8 + i] = kq + __shfl_xor_sync(0xffffffffu, sq, 4);
			}
			float r2[8];
			const bool hi2 = rl & 2;
#pragma unroll
			for (int i = 0; i < 4; i++) {
				const float sw = hi2 ? r1[i] : r1[4 + i], kw = hi2 ? r1[4 + i] : r1[i];
				const float sq = hi2 ? r1[8 + i] : r1[12 + i], kq = hi2 ? r1[12 + i] : r1[8 + i];
				r2[i] = kw + __shfl_xor_sync(0xffffffffu, sw, 2);
				r2[4 + i] = kq + __shfl_xor_sync(0xffffffffu, sq, 2);
			}
			const bool hi1 = rl & 1;
#pragma unroll
			for (int i = 0; i < 2; i++) {
				const float sw = hi1 ? r2[i] : r2[2 + i], kw = hi1 ? r2[2 + i] : r2[i];
				const float sq = hi1 ? r2[4 + i] : r2[6 + i], kq = hi1 ? r2[6 + i] : r2[4 + i];
				w2[i] = kw + __shfl_xor_sync(0xffffffffu, sw, 1);
				q2[i] = kq + __shfl_xor_sync(0xffffffffu, sq, 1);
			}
		}
		const int vc = warp * 4 + (lane >> 3);
		float u2[2];
		u2[0] = sV[(2 * rl) * 16 + vc] - w2[0];
		u2[1] = sV[(2 * rl + 1) * 16 + vc] - w2[1];
		// every lane needs all of the column's u
		float u[DB];
#pragma unroll
		for (int t = 0; t < DB; t++) u[t] = __shfl_sync(0xffffffffu, u2[t & 1], (lane & 24) + (t >> 1));
		if (on) {
#pragma unroll
			for (int i = 0; i < 2; i++) {
				const int t = 2 * rl + i;
				float o = q2[i];
#pragma unroll
				for (int s = 0; s < DB; s++) o = fmaf(sM[t * DB + s], u[s], o);  // (zero above the diagonal)
				if (b * DB + t < len) a.o[size_t(row0 + b * DB + t) * a.H * dv + h * dv + c] = o;
			}
		}
#pragma unroll
		for (int j = 0; j < RPL / 4; j++) {
			const float4 g = *reinterpret_cast<const float4 *>(sD + 4 * rl + 32 * j);
			S[4 * j] *= g.x; S[4 * j + 1] *= g.y; S[4 * j + 2] *= g.z; S[4 * j + 3] *= g.w;
		}
#pragma unroll
		for (int t = 0; t < DB; t++)
#pragma unroll
			for (int j = 0; j < RPL / 4; j++) {
				const float4 k = *reinterpret_cast<const float4 *>(sK + t * DKP + 4 * rl + 32 * j);
				S[4 * j] = fmaf(k.x, u[t], S[4 * j]); S[4 * j + 1] = fmaf(k.y, u[t], S[4 * j + 1]);
				S[4 * j + 2] = fmaf(k.z, u[t], S[4 * j + 2]); S[4 * j + 3] = fmaf(k.w, u[t], S[4 * j + 3]);
			}
		__syncthreads();
	}
#pragma unroll
	for (int j = 0; j < RPL; j++) {
		const int i = 4 * rl + 32 * (j >> 2) + (j & 3);
		if (on && i < dk) Sg[size_t(i) * dv + c] = S[j];
	}
}
template <int RPL> constexpr size_t delta_scan_smem() { return size_t(2) * (3 * DB * 8 * RPL + 8 * RPL + DB * DB + DB * 16) * 4; }

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
