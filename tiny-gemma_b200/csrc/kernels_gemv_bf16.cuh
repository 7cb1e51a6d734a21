// Matrix-vector products with bfloat16 weights [N][K] for a few rows (decoding): HBM bound. Activations stay fp32.
// The norm (and input convolution) that precedes a product is its prologue, what follows it is its epilogue. A layer
// whose feed-forward follows its mixer is five launches: [norm + conv -> projections -> cache], token mixing, [output
// projection + residual], [norm -> gate|up -> gated activation], [down + residual]. A layer whose feed-forward stands
// beside its mixer is three (GV_FRONT, token mixing, GV_MIX): [norm + shift -> projections, gate|up -> gated activation,
// router], token mixing beside the chosen experts' gate|up (kernels_moe.cuh), [read-out norm and gate -> output
// projection, down, the experts' down + residual].
//
// A CTA of 8 warps walks groups of output rows: a warp owns NR rows of the group (or, with KS > 1, the KS warps of a
// row set share its K range), a lane 8 consecutive k of every 256. The next 16-byte weight words are requested before
// the current ones are used, the very first ones before the wait for the preceding kernel.
#pragma once
#include "kernels_gemm_bf16.cuh"
#include "kernels_rowwise.cuh"

namespace tg {

enum GemvPro { GV_VEC = 0, GV_LN = 1, GV_LN_CONV = 2, GV_MIX = 3 };
enum GemvEpi { GV_PROJ = 0, GV_ADD = 1, GV_GLU = 2, GV_LOGITS = 3, GV_FRONT = 4 };
// what GV_MIX does to a mixer's raw read-out
enum MixNorm { MIX_NONE = 0, MIX_GATE_NORM = 1 /* norm(o silu(z)) w */, MIX_NORM_GATE = 2 /* norm(o) w sigmoid(z) */ };

struct GemvArgs {
	StepDesc d;
	const __nv_bfloat16 *W;
	int ldw, N, K;             // K: columns that are used (a multiple of 8; surplus columns and activations are zero)
	const float *vec;          // GV_VEC: [R][ldv]
	int ldv;
	const float *x;            // residual stream [R][ldx]
	int ldx, D;
	const __nv_bfloat16 *embed;
	int lde, V;
	int embed_mode;            // 0: x; 1: x = embed[tok] (nothing written there yet); 2: x + embed[tok]
	const float *w;            // norm weight [D]
	float eps;
	const float *cw;           // convolution [taps][D]
	float *hist;               // [B][2][taps-1][D]
	int taps;
	float *out;                // GV_PROJ, GV_GEGLU, GV_LOGITS: [R][ldo]; GV_ADD: the residual stream [R][ldo]
	int ldo;
	float *norm_out;           // normed rows [R][D], written by one CTA, or null
	float cap;
	// GV_PROJ: columns p_k .. and p_v .. also go to the cache
	int p_k, n_k, p_v, n_v;
	void *kc, *vc, *ks, *vs;
	int cap_rows, keep, keep_rows, cache_f32;
	int *err;
	int rms;                   // the norm takes off no mean
	float embed_scale;
	int act;                   // gated activation
	float limit;
	// GV_FRONT: weight rows are [n_proj of the projections][2 n_glu gate | up][n_route router rows]; the projections read
	// the convolved norm, the others the plain one. Projection columns from n32 on go to out32.
	int n_proj, n32, n_glu, n_route;
	float *out32;
	int ld32;
	float *glu_out, *route_out;
	int ld_glu, ld_route;
	// GV_MIX: columns 0 .. mix_n-1 of vec are a raw read-out, `parts` equal parts of it normed
	int mix_norm, mix_n, parts;
	const float *gate;         // [R][ldg]
	int ldg;
	// chosen experts: activations [R][top][n_ex], their weights and ids [R][top], down projections [experts][N][ld_ex]
	const float *ex_act, *ex_w;
	const int *ex_id;
	int top, n_ex, ld_ex;
	const __nv_bfloat16 *ex_W;
};

constexpr int GV_THREADS = 256;
__host__ __device__ inline int gv_k8(int K) { return (K + 7) / 8; }
template <int R, int NR> __host__ __device__ constexpr int gv_red_floats() { return 2 * 8 * NR * R; }
template <int R, int NR> size_t gv_smem(int K, int pro, int epi, int parts, int top, int ex) {
	const size_t rows = epi == GV_FRONT ? 2 * R : R, extra = pro == GV_LN ? 1 : (pro == GV_LN_CONV ? 1 + R : 0);
	return ((rows + extra) * 8 * gv_k8(K) + gv_red_floats<R, NR>() + 32 + (pro == GV_MIX ? size_t(R) * ((parts + 3) / 4 * 4 + ex + top) : 0)) * 4;
}

// sum over the threads of a row (8 / R warps), in every one of them
template <int R> __device__ __forceinline__ float gv_row_sum(float v, float *red) {
	v = warp_sum(v);
	__syncthreads();
	if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
	__syncthreads();
	const float *mine = red + (threadIdx.x >> 5) / (8 / R) * (8 / R);
	float t = 0.0f;
#pragma unroll
	for (int w = 0; w < 8 / R; w++) t += mine[w];
	return t;
}

template <int R, int NR, int KS, int PRO, int EPI>
__global__ void __launch_bounds__(GV_THREADS) gemv_bf16_kernel(GemvArgs a) {
	pdl_trigger();
	extern __shared__ __align__(16) float gv_sm[];
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int K8 = gv_k8(a.K);
	float *xs = gv_sm;                                   // [R][two halves of 8 k][K8] float4
	float *red = gv_sm + size_t(R) * 8 * K8;             // [2][row set][KS][NR][R]
	float *bred = red + gv_red_floats<R, NR>();
	float *wn = bred + 32, *hc = wn + 8 * K8;            // norm weight (x its factor in the convolution); history's share
	float *xp = hc + size_t(R) * 8 * K8;                 // GV_FRONT: the plain norms, laid out as xs
	float *prt = bred + 32, *xe = prt + (PRO == GV_MIX ? R * ((a.parts + 3) / 4 * 4) : 0);  // GV_MIX: 1 / deviation of the parts; experts' activations
	int *xid = reinterpret_cast<int *>(xe + (PRO == GV_MIX ? R * a.top * a.n_ex : 0));  // the rows' chosen experts
	constexpr int SETS = 8 / KS, GROUP = SETS * NR;      // weight rows per CTA and group
	const int set = warp / KS, ks = warp % KS;
	const int n_out = EPI == GV_GLU ? a.N / 2 : (EPI == GV_LOGITS ? a.ldo : a.N);
	constexpr int OUTS = EPI == GV_GLU ? GROUP / 2 : GROUP;  // outputs per group
	const int gp = EPI == GV_FRONT ? (a.n_proj + GROUP - 1) / GROUP : 0, gg = EPI == GV_FRONT ? gp + (a.n_glu + GROUP / 2 - 1) / (GROUP / 2) : 0;
	const int groups = EPI == GV_FRONT ? gg + (a.n_route + GROUP - 1) / GROUP : (n_out + OUTS - 1) / OUTS;
	const int nit = (K8 + 32 * KS - 1) / (32 * KS);

	// weight row i (of NR) of this warp in a group
	auto wrow = [&](int grp, int i) -> int {
		if (EPI == GV_FRONT) {
			if (grp < gp) {
				const int n = grp * GROUP + set * NR + i;
				return n < a.n_proj ? n : a.N;
			}
			if (grp < gg) {
				const int o = (grp - gp) * (GROUP / 2) + set * (NR / 2) + (i >> 1);
				return o < a.n_glu ? a.n_proj + (o >> 4) * 32 + (o & 15) + (i & 1) * 16 : a.N;
			}
			const int n = (grp - gg) * GROUP + set * NR + i;
			return n < a.n_route ? a.n_proj + 2 * a.n_glu + n : a.N;
		}
		if (EPI == GV_GLU) {
			const int o = grp * OUTS + set * (NR / 2) + (i >> 1);
			return (o >> 4) * 32 + (o & 15) + (i & 1) * 16;
		}
		return grp * GROUP + set * NR + i;
	};
	auto load = [&](int grp, int it, uint4 (&w)[NR]) {
		const int k8 = (it * KS + ks) * 32 + lane;
#pragma unroll
		for (int i = 0; i < NR; i++) {
			const int n = wrow(grp, i);
			w[i] = make_uint4(0, 0, 0, 0);
			if (grp < groups && n < a.N && k8 < K8) {
				const int4 v = ld_stream_int4(a.W + size_t(n) * a.ldw + 8 * k8);
				w[i] = make_uint4(v.x, v.y, v.z, v.w);
			}
		}
	};
	uint4 cur[NR], nxt[NR];
	load(blockIdx.x, 0, cur);
	if (PRO == GV_LN || PRO == GV_LN_CONV) {  // (weights too: nobody's output)
#pragma unroll 4
		for (int k = tid; k < a.D; k += GV_THREADS) wn[k] = PRO == GV_LN_CONV ? fmaf(a.cw[size_t(a.taps - 1) * a.D + k], a.w[k], a.w[k]) : a.w[k];
	}
	pdl_wait();

	// ---------------------------------------------------------------- prologue: activations into shared memory
	// (the rows side by side, TG threads each; global loads in batches of four, ahead of the stores)
	auto xi = [&](int k) { return ((k >> 2) & 1) * 4 * K8 + (k >> 3) * 4 + (k & 3); };
	constexpr int TG = GV_THREADS / R;
	const int r = tid / TG, t = tid % TG;
	float *xr = xs + size_t(r) * 8 * K8;
	if constexpr (PRO == GV_VEC || PRO == GV_MIX) {
		const float *vec = a.vec + size_t(r) * a.ldv, *gate = PRO == GV_MIX ? a.gate + size_t(r) * a.ldg : nullptr;
		const bool pre = PRO == GV_MIX && a.mix_norm == MIX_GATE_NORM;
		for (int u0 = t; u0 < 2 * K8; u0 += 4 * TG) {  // (K is a multiple of 8)
			float4 v[4], z[4];
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const int u = u0 + e * TG;
				if (u < 2 * K8) v[e] = *reinterpret_cast<const float4 *>(vec + 4 * u);
				if (pre && 4 * u < a.mix_n) z[e] = *reinterpret_cast<const float4 *>(gate + 4 * u);
			}
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const int u = u0 + e * TG, k = 4 * u;
				if (u >= 2 * K8) break;
				if (pre) {
					if (k < a.mix_n) v[e].x *= silu_f(z[e].x);
					if (k + 1 < a.mix_n) v[e].y *= silu_f(z[e].y);
					if (k + 2 < a.mix_n) v[e].z *= silu_f(z[e].z);
					if (k + 3 < a.mix_n) v[e].w *= silu_f(z[e].w);
				}
				*reinterpret_cast<float4 *>(xr + xi(k)) = v[e];
			}
		}
		if (PRO == GV_MIX) {
			const int n4 = a.n_ex / 4, all4 = a.top * n4;
			float4 *dst = reinterpret_cast<float4 *>(xe + r * a.top * a.n_ex);
			const float4 *src = reinterpret_cast<const float4 *>(a.ex_act + size_t(r) * a.top * a.n_ex);
			const float *ew = a.ex_w + r * a.top;
			for (int u = t; u < a.top; u += TG) xid[r * a.top + u] = a.ex_id[r * a.top + u];
#pragma unroll 4
			for (int u = t; u < all4; u += TG) {
				const float4 v = src[u];
				const float w = ew[u / n4];
				dst[u] = make_float4(v.x * w, v.y * w, v.z * w, v.w * w);
			}
			if (a.mix_norm != MIX_NONE) {
				__syncthreads();
				const int width = a.mix_n / a.parts;
				for (int p = warp % (8 / R); p < a.parts; p += 8 / R) {
					float q = 0.0f;
#pragma unroll 4
					for (int k = p * width + lane; k < (p + 1) * width; k += 32) q = fmaf(xr[xi(k)], xr[xi(k)], q);
					q = warp_sum(q);
					if (lane == 0) prt[r * a.parts + p] = 1.0f / sqrtf(q / float(width) + a.eps);
				}
				__syncthreads();
				const bool post = a.mix_norm == MIX_NORM_GATE;
#pragma unroll 4
				for (int k = t; k < a.mix_n; k += TG) {
					const float w = a.w[k], z = post ? gate[k] : 0.0f;
					const float v = xr[xi(k)] * prt[r * a.parts + k / width] * w;
					xr[xi(k)] = post ? v * sigmoid_f(z) : v;
				}
			}
		}
	} else {
		const int seg = a.d.row_seg[r];
		int tok = 0;
		if (a.embed_mode) {
			tok = a.d.tok[r];
			if (tok < 0 || tok >= a.V) {
				if (blockIdx.x == 0 && t == 0) *a.err = 1;
				tok = 0;
			}
		}
		const int H = PRO == GV_LN_CONV ? a.taps - 1 : 0;
		const float *hr = nullptr;
		float *hw = nullptr, *hcr = hc + size_t(r) * 8 * K8;
		int pos = 0;
		if (PRO == GV_LN_CONV) {
			pos = a.d.seg_pos[seg];
			float *hb = a.hist + size_t(a.d.seg_seq[seg]) * 2 * H * a.D;
			hr = hb + size_t(a.d.seg_par[seg]) * H * a.D;
			hw = hb + size_t(a.d.seg_par[seg] ^ 1) * H * a.D;
		}
		float s = 0.0f;
		for (int k0 = t; k0 < a.D; k0 += 4 * TG) {
			float v[4], c[4] = {}, em[4];
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const int k = k0 + e * TG;
				v[e] = k < a.D && a.embed_mode != 1 ? a.x[size_t(r) * a.ldx + k] : 0.0f;
				em[e] = k < a.D && a.embed_mode ? __bfloat162float(a.embed[size_t(tok) * a.lde + k]) : 0.0f;
			}
			if (PRO == GV_LN_CONV) {
				for (int j = 0; j < H; j++) {
					float u[4], w[4];
#pragma unroll
					for (int e = 0; e < 4; e++) {
						const int k = k0 + e * TG;
						u[e] = k < a.D && pos - H + j >= 0 ? hr[size_t(j) * a.D + k] : 0.0f;
						w[e] = k < a.D ? a.cw[size_t(j) * a.D + k] : 0.0f;
					}
#pragma unroll
					for (int e = 0; e < 4; e++) {
						c[e] = fmaf(w[e], u[e], c[e]);
						if (blockIdx.x == 0 && j > 0 && k0 + e * TG < a.D) hw[size_t(j - 1) * a.D + k0 + e * TG] = u[e];
					}
				}
			}
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const int k = k0 + e * TG;
				if (k >= a.D) break;
				v[e] = fmaf(a.embed_scale, em[e], v[e]);
				if (PRO == GV_LN_CONV) hcr[k] = c[e];
				xr[xi(k)] = v[e];
				s += v[e];
			}
		}
		const float mean = a.rms ? 0.0f : gv_row_sum<R>(s, bred) / float(a.D);
		float q = 0.0f;
		for (int k = t; k < a.D; k += TG) {
			const float c = xr[xi(k)] - mean;
			q = fmaf(c, c, q);
		}
		const float rstd = 1.0f / sqrtf(gv_row_sum<R>(q, bred) / float(a.D) + a.eps);
		for (int k0 = t; k0 < 8 * K8; k0 += 4 * TG) {
			float w[4];
#pragma unroll
			for (int e = 0; e < 4; e++) w[e] = PRO == GV_LN_CONV && k0 + e * TG < a.D ? a.w[k0 + e * TG] : 0.0f;
#pragma unroll
			for (int e = 0; e < 4; e++) {
				const int k = k0 + e * TG;
				if (k >= 8 * K8) break;
				float y = 0.0f, plain = 0.0f;
				if (k < a.D) {
					const float n = (xr[xi(k)] - mean) * rstd;
					plain = n * w[e];
					y = n * wn[k];
					if (PRO == GV_LN_CONV) {
						y += hcr[k];
						if (blockIdx.x == 0 && H > 0) hw[size_t(H - 1) * a.D + k] = plain;
					}
					if (a.norm_out && blockIdx.x == 0) a.norm_out[size_t(r) * a.D + k] = EPI == GV_FRONT ? plain : y;
				}
				if (EPI == GV_FRONT) xp[size_t(r) * 8 * K8 + xi(k)] = plain;
				xr[xi(k)] = y;
			}
		}
	}
	__syncthreads();

	// ---------------------------------------------------------------- products
	int flip = 0;
	for (int grp = blockIdx.x; grp < groups; grp += gridDim.x, flip ^= 1) {
		float acc[R][NR] = {};
		const float *xg = EPI == GV_FRONT && grp >= gp ? xp : xs;
		for (int it = 0; it < nit; it++) {
			if (it + 1 < nit) load(grp, it + 1, nxt);
			else load(grp + gridDim.x, 0, nxt);
			const int k8 = (it * KS + ks) * 32 + lane;
			if (k8 < K8) {
#pragma unroll
				for (int r = 0; r < R; r++) {
					const float4 x0 = *reinterpret_cast<const float4 *>(xg + size_t(r) * 8 * K8 + 4 * k8);
					const float4 x1 = *reinterpret_cast<const float4 *>(xg + size_t(r) * 8 * K8 + 4 * K8 + 4 * k8);
#pragma unroll
					for (int i = 0; i < NR; i++) {
						float s = acc[r][i];
						s = fmaf(bf16_lo(cur[i].x), x0.x, s);
						s = fmaf(bf16_hi(cur[i].x), x0.y, s);
						s = fmaf(bf16_lo(cur[i].y), x0.z, s);
						s = fmaf(bf16_hi(cur[i].y), x0.w, s);
						s = fmaf(bf16_lo(cur[i].z), x1.x, s);
						s = fmaf(bf16_hi(cur[i].z), x1.y, s);
						s = fmaf(bf16_lo(cur[i].w), x1.z, s);
						acc[r][i] = fmaf(bf16_hi(cur[i].w), x1.w, s);
					}
				}
			}
#pragma unroll
			for (int i = 0; i < NR; i++) cur[i] = nxt[i];
		}
		if (PRO == GV_MIX && a.top) {  // each row's own experts: 16 bytes of (expert, k) per lane, the rows' loads together
			const int e8 = a.n_ex / 8, n0 = grp * GROUP + set * NR;
			for (int j = ks * 32 + lane; j < a.top * e8; j += 32 * KS) {
				const int k = j / e8, o = 8 * (j % e8);
				int4 w[R][NR];
#pragma unroll
				for (int r = 0; r < R; r++) {
					const __nv_bfloat16 *W = a.ex_W + size_t(xid[r * a.top + k]) * a.N * a.ld_ex + o;
#pragma unroll
					for (int i = 0; i < NR; i++) w[r][i] = n0 + i < a.N ? ld_stream_int4(W + size_t(n0 + i) * a.ld_ex) : make_int4(0, 0, 0, 0);
				}
#pragma unroll
				for (int r = 0; r < R; r++) {
					const float *xv = xe + r * a.top * a.n_ex + 8 * j;
					const float4 x0 = *reinterpret_cast<const float4 *>(xv), x1 = *reinterpret_cast<const float4 *>(xv + 4);
#pragma unroll
					for (int i = 0; i < NR; i++) {
						const int4 &v = w[r][i];
						float s = acc[r][i];
						s = fmaf(bf16_lo(v.x), x0.x, s);
						s = fmaf(bf16_hi(v.x), x0.y, s);
						s = fmaf(bf16_lo(v.y), x0.z, s);
						s = fmaf(bf16_hi(v.y), x0.w, s);
						s = fmaf(bf16_lo(v.z), x1.x, s);
						s = fmaf(bf16_hi(v.z), x1.y, s);
						s = fmaf(bf16_lo(v.w), x1.z, s);
						acc[r][i] = fmaf(bf16_hi(v.w), x1.w, s);
					}
				}
			}
		}
		float *rb = red + flip * 8 * NR * R;
#pragma unroll
		for (int i = 0; i < NR; i++)
#pragma unroll
			for (int r = 0; r < R; r++) {
				const float v = warp_sum(acc[r][i]);
				if (lane == 0) rb[((set * KS + ks) * NR + i) * R + r] = v;
			}
		__syncthreads();
		// one thread per (output, row); the other copy of `red` keeps the next group from overwriting it
		if (tid < OUTS * R) {
			const int o = tid / R, r = tid % R, n = grp * OUTS + o;
			auto sum = [&](int st, int i) {
				float v = 0.0f;
#pragma unroll
				for (int q = 0; q < KS; q++) v += rb[((st * KS + q) * NR + i) * R + r];
				return v;
			};
			if (EPI == GV_FRONT) {
				if (grp < gp) {
					const float v = sum(o / NR, o % NR);
					if (n < a.n32) a.out[size_t(r) * a.ldo + n] = v;
					else if (n < a.n_proj) a.out32[size_t(r) * a.ld32 + n - a.n32] = v;
				} else if (grp < gg) {
					const int st = o / (NR / 2), i = (o % (NR / 2)) * 2, c = (grp - gp) * (GROUP / 2) + o;
					if (o < GROUP / 2 && c < a.n_glu) a.glu_out[size_t(r) * a.ld_glu + c] = glu(a.act, a.limit, sum(st, i), sum(st, i + 1));
				} else {
					const int c = (grp - gg) * GROUP + o;
					if (c < a.n_route) a.route_out[size_t(r) * a.ld_route + c] = sum(o / NR, o % NR);
				}
			} else if (n < n_out) {
				float *dst = a.out + size_t(r) * a.ldo + n;
				if (EPI == GV_GLU) {
					const int st = o / (NR / 2), i = (o % (NR / 2)) * 2;
					*dst = glu(a.act, a.limit, sum(st, i), sum(st, i + 1));
				} else {
					const float v = sum(o / NR, o % NR);
					if (EPI == GV_ADD) {
						float b = a.embed_mode == 1 ? 0.0f : *dst;
						if (a.embed_mode) b += a.embed_scale * __bfloat162float(a.embed[size_t(min(max(a.d.tok[r], 0), a.V - 1)) * a.lde + n]);
						*dst = b + v;
					} else if (EPI == GV_LOGITS) {
						*dst = n < a.N ? soft_cap(v, a.cap) : -INFINITY;
					} else {
						*dst = v;
						const bool isk = n >= a.p_k && n < a.p_k + a.n_k, isv = n >= a.p_v && n < a.p_v + a.n_v;
						if (isk || isv) {
							const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], pos = a.d.seg_pos[seg];
							const int w = isk ? a.n_k : a.n_v, c = n - (isk ? a.p_k : a.p_v);
							const size_t ring = (size_t(seq) * a.cap_rows + pos % a.cap_rows) * w + c, first = (size_t(seq) * a.keep_rows + pos) * w + c;
							void *rp = isk ? a.kc : a.vc, *fp = isk ? a.ks : a.vs;
							if (a.cache_f32) {
								reinterpret_cast<float *>(rp)[ring] = v;
								if (pos < a.keep) reinterpret_cast<float *>(fp)[first] = v;
							} else {
								reinterpret_cast<__nv_bfloat16 *>(rp)[ring] = __float2bfloat16_rn(v);
								if (pos < a.keep) reinterpret_cast<__nv_bfloat16 *>(fp)[first] = __float2bfloat16_rn(v);
							}
						}
					}
				}
			}
		}
	}
}

}  // namespace tg
