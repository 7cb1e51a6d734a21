// Causal attention over a sliding window plus the first tokens of a sequence, with an optional per-head distance
// bias taken off the scores:
//     score(i, j) = scale * q_i . k_j - r1 ln(1 + r2 (i - j)),     j <= i and (i - j < window or j < keep_first)
// or, instead of the first tokens, pooled blocks: for each block of `pool` tokens that lies wholly before the window one
// row, the mean of the block's cached keys and of its values. Grouped key/value heads; an optional sigmoid output gate;
// optional rotation of q and k and norm of v, applied between the projections and the cache.
//
// Cache of one layer run, per sequence: a ring of `cap` rows (slot = position mod cap; cap is a multiple of 64 and at
// least window + rows of a step) and, because the ring forgets them, a second store: a copy of the first keep_first rows,
// or the pooled rows (block b at row b, written when its last token arrives). A query takes keys within its window from
// the ring and the others from the second store, so no key is met twice.
// Rows hold G heads one after the other, each padded to a multiple of 16 elements (dkp, dvp) with zeros.
//
//   kv_append_kernel        rows of a step -> cache
//   kv_transform_kernel     the same with rotation, value norm and pooling
//   window_attn_kernel      portions, CUDA cores: any sizes, fp32 or bf16
//   window_attn_tc_kernel   portions, bf16 on tcgen05 (dkp, dvp <= 256): 128 queries of one head per CTA
//   window_attn_token_cta   one token per sequence: a CTA per (sequence, key/value head, run of keys)
#pragma once
#include "kernels_gemm_bf16.cuh"
#include "kernels_rowwise.cuh"

namespace tg {

struct WAttnArgs {
	StepDesc d;
	int H, G, dk, dv, dkp, dvp;
	float scale;
	int window, keep;      // keep: first tokens that stay visible
	int pool;              // tokens of a pooled block (0: none; then keep = 0)
	int rot;               // rotated dimensions of q and k, pair (c, c + rot/2) (0: none)
	const float2 *cs;      // [R][ld_cs] cos and sin of the rows' positions
	int ld_cs;
	int vnorm;             // values are divided by their root mean square
	float eps;
	int append;            // one token per sequence: the token's key and value still have to be put into the cache
	const float *r1, *r2;  // [H] or null
	const void *p;         // projections, rows of ldp: q at p_q, k at p_k, v at p_v, gate at p_g (-1: none)
	int ldp, p_q, p_k, p_v, p_g;
	void *kc, *vc;         // [B][cap][G*dkp], [B][cap][G*dvp]
	void *ks, *vs;         // [B][keep_rows][G*dkp], ...: the first tokens, or the pooled blocks
	int cap, keep_rows;    // keep_rows: rows of the second store, a multiple of 64
	void *out;             // [R] rows of ldo, head h at h*dvp
	int ldo;
	float out_scale;
	// one token per sequence: partial results of the runs of keys
	float *part;           // [B][G][nsplit][per][dvp + 2]
	unsigned *tickets;     // [B][G], zero between launches
	int nsplit;
	int *err;
};

template <typename PT, typename CT>
static __global__ void __launch_bounds__(256) kv_append_kernel(WAttnArgs a) {
	pdl_trigger();
	pdl_wait();
	const int r = blockIdx.x, seg = a.d.row_seg[r], seq = a.d.seg_seq[seg];
	const int pos = a.d.seg_pos[seg] + r - a.d.seg_row[seg], slot = pos % a.cap;
	const PT *row = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	const int nk = a.G * a.dkp, nv = a.G * a.dvp;
	for (int i = threadIdx.x; i < nk + nv; i += 256) {
		const bool isk = i < nk;
		const int c = isk ? i : i - nk, n = isk ? nk : nv;
		const CT v = from_f32<CT>(to_f32(row[(isk ? a.p_k : a.p_v) + c]));
		reinterpret_cast<CT *>(isk ? a.kc : a.vc)[(size_t(seq) * a.cap + slot) * n + c] = v;
		if (pos < a.keep) reinterpret_cast<CT *>(isk ? a.ks : a.vs)[(size_t(seq) * a.keep_rows + pos) * n + c] = v;
	}
}

// element c of a rotated head
template <typename PT> __device__ __forceinline__ float wa_rotated(const WAttnArgs &a, const PT *head, const float2 *cs, int c) {
	const float u = to_f32(head[c]);
	const int half = a.rot >> 1;
	if (c >= a.rot) return u;
	if (c < half) return u * cs[c].x - to_f32(head[c + half]) * cs[c].y;
	return u * cs[c - half].x + to_f32(head[c - half]) * cs[c - half].y;
}
// the mean of block b of the ring -> row b of the second store; NT threads, this one is number t
template <typename CT, int NT> __device__ __forceinline__ void wa_pool_block(const WAttnArgs &a, int seq, int g, int b, int t) {
	const int nk = a.G * a.dkp, nv = a.G * a.dvp;
	for (int c = t; c < a.dkp + a.dvp; c += NT) {
		const bool isk = c < a.dkp;
		const int n = isk ? nk : nv, col = isk ? g * a.dkp + c : g * a.dvp + c - a.dkp;
		const CT *ring = reinterpret_cast<const CT *>(isk ? a.kc : a.vc) + size_t(seq) * a.cap * n + col;
		float s = 0.0f;
		const int first = (b * a.pool) % a.cap, wrap = a.cap - first;  // (row j lies at slot first + j, or that minus cap)
#pragma unroll 8
		for (int j = 0; j < a.pool; j++) s += to_f32(ring[size_t(first + j - (j >= wrap ? a.cap : 0)) * n]);
		reinterpret_cast<CT *>(isk ? a.ks : a.vs)[(size_t(seq) * a.keep_rows + b) * n + col] = from_f32<CT>(s / float(a.pool));
	}
}
__device__ __forceinline__ float2 load2(const float *p) { return *reinterpret_cast<const float2 *>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16 *p) {
	const uint32_t u = *reinterpret_cast<const uint32_t *>(p);
	return make_float2(bf16_lo(u), bf16_hi(u));
}
__device__ __forceinline__ void store2(float *p, float2 v) { *reinterpret_cast<float2 *>(p) = v; }
__device__ __forceinline__ void store2(__nv_bfloat16 *p, float2 v) { *reinterpret_cast<uint32_t *>(p) = pack_bf16(v.x, v.y); }
// Portions: rotates q in place, puts rotated keys and normed values into the ring, and pools the blocks that the step
// completes. A CTA owns `unit` positions (a multiple of `pool`, counted from the sequence's start) of a key/value head, so
// that what a block needs is either its own or an earlier step's. grid (units of the longest segment + 1, G, segments)
template <typename PT, typename CT>
static __global__ void __launch_bounds__(256) kv_transform_kernel(WAttnArgs a, int unit) {
	pdl_trigger();
	pdl_wait();
	const int seg = blockIdx.z, g = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int pos = a.d.seg_pos[seg], len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], seq = a.d.seg_seq[seg];
	const int u0 = (pos / unit + int(blockIdx.x)) * unit;
	if (u0 >= pos + len) return;
	const int lo = max(pos, u0), hi = min(pos + len, u0 + unit), per = a.H / a.G, half = a.rot >> 1;
	const int nk = a.G * a.dkp, nv = a.G * a.dvp;
	for (int i = lo + warp; i < hi; i += 8) {
		const int r = row0 + i - pos;
		PT *row = const_cast<PT *>(reinterpret_cast<const PT *>(a.p)) + size_t(r) * a.ldp;
		const float2 *cs = a.cs + size_t(r) * a.ld_cs;
		PT *q0 = row + a.p_q + g * per * a.dkp;
		if (half % 2 == 0) {
			for (int c = 2 * lane; c < half; c += 64) {
				const float4 t = *reinterpret_cast<const float4 *>(cs + c);  // cos, sin, cos, sin
#pragma unroll 4
				for (int h = 0; h < per; h++) {
					PT *q = q0 + h * a.dkp + c;
					const float2 u = load2(q), v = load2(q + half);
					store2(q, make_float2(u.x * t.x - v.x * t.y, u.y * t.z - v.y * t.w));
					store2(q + half, make_float2(v.x * t.x + u.x * t.y, v.y * t.z + u.y * t.w));
				}
			}
		} else {
			for (int c = lane; c < half; c += 32)
				for (int h = 0; h < per; h++) {
					PT *q = q0 + h * a.dkp + c;
					const float u = to_f32(q[0]), v = to_f32(q[half]);
					q[0] = from_f32<PT>(u * cs[c].x - v * cs[c].y);
					q[half] = from_f32<PT>(v * cs[c].x + u * cs[c].y);
				}
		}
		const size_t slot = size_t(seq) * a.cap + i % a.cap;
		CT *kd = reinterpret_cast<CT *>(a.kc) + slot * nk + g * a.dkp, *vd = reinterpret_cast<CT *>(a.vc) + slot * nv + g * a.dvp;
		const PT *ks = row + a.p_k + g * a.dkp, *vs = row + a.p_v + g * a.dvp;
		if (half % 2 == 0) {
			for (int c = 2 * lane; c < half; c += 64) {
				const float4 t = *reinterpret_cast<const float4 *>(cs + c);
				const float2 u = load2(ks + c), v = load2(ks + half + c);
				store2(kd + c, make_float2(u.x * t.x - v.x * t.y, u.y * t.z - v.y * t.w));
				store2(kd + half + c, make_float2(v.x * t.x + u.x * t.y, v.y * t.z + u.y * t.w));
			}
			for (int c = a.rot + 2 * lane; c < a.dkp; c += 64) store2(kd + c, load2(ks + c));
		} else {
			for (int c = lane; c < a.dkp; c += 32) kd[c] = from_f32<CT>(wa_rotated(a, ks, cs, c));
		}
		float f = 1.0f;
		if (a.vnorm) {  // (padding columns are zero)
			float s = 0.0f;
			for (int c = 2 * lane; c < a.dvp; c += 64) {
				const float2 v = load2(vs + c);
				s = fmaf(v.x, v.x, fmaf(v.y, v.y, s));
			}
			f = 1.0f / sqrtf(warp_sum(s) / float(a.dv) + a.eps);
		}
		for (int c = 2 * lane; c < a.dvp; c += 64) {
			const float2 v = load2(vs + c);
			store2(vd + c, make_float2(v.x * f, v.y * f));
		}
	}
	if (!a.pool) return;
	__syncthreads();
	for (int b = u0 / a.pool; (b + 1) * a.pool <= hi; b++)
		if ((b + 1) * a.pool > pos) wa_pool_block<CT, 256>(a, seq, g, b, tid);
}

// number of keys a query at position i sees, and key number n -> position
__device__ __forceinline__ int wa_first(const WAttnArgs &a, int i) { return max(0, i - a.window + 1); }      // first window position
// rows of the second store that it sees: kept tokens outside the window, or blocks whose last token has left it
__device__ __forceinline__ int wa_kept(const WAttnArgs &a, int i) {
	return a.pool ? max(0, (i - a.window + 1) / a.pool) : min(a.keep, wa_first(a, i));
}
__device__ __forceinline__ float wa_bias(float r1, float r2, int dist) { return r1 * log1pf(r2 * float(dist)); }

// ------------------------------------------------------------------ portions, CUDA cores
// One warp per (row, head); a lane scores one key of 32, then the lanes own the value dimensions.
template <typename PT, typename CT>
static __global__ void __launch_bounds__(128) window_attn_kernel(WAttnArgs a, int R) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ float wa_sm[];
	const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
	const int item = blockIdx.x * 4 + warp;
	float *q = wa_sm + warp * (a.dkp + a.dvp), *o = q + a.dkp;
	if (item >= R * a.H) return;
	const int r = item / a.H, h = item % a.H, g = h / (a.H / a.G);
	const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], i = a.d.seg_pos[seg] + r - a.d.seg_row[seg];
	const PT *row = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	for (int c = lane; c < a.dkp; c += 32) q[c] = to_f32(row[a.p_q + h * a.dkp + c]) * a.scale;
	for (int c = lane; c < a.dvp; c += 32) o[c] = 0.0f;
	__syncwarp();
	const CT *kc = reinterpret_cast<const CT *>(a.kc) + size_t(seq) * a.cap * a.G * a.dkp, *vc = reinterpret_cast<const CT *>(a.vc) + size_t(seq) * a.cap * a.G * a.dvp;
	const CT *ks = reinterpret_cast<const CT *>(a.ks) + size_t(seq) * a.keep_rows * a.G * a.dkp, *vs = reinterpret_cast<const CT *>(a.vs) + size_t(seq) * a.keep_rows * a.G * a.dvp;
	const int first = wa_first(a, i), kept = wa_kept(a, i), total = kept + i - first + 1;
	const float r1 = a.r1 ? a.r1[h] : 0.0f, r2 = a.r2 ? a.r2[h] : 0.0f;
	float m = -INFINITY, l = 0.0f;
	for (int n0 = 0; n0 < total; n0 += 32) {
		const int n = n0 + lane;
		float s = -INFINITY;
		if (n < total) {
			const int j = n < kept ? n : first + n - kept;
			const CT *k = n < kept ? ks + size_t(j) * a.G * a.dkp + g * a.dkp : kc + size_t(j % a.cap) * a.G * a.dkp + g * a.dkp;
			s = 0.0f;
			for (int c = 0; c < a.dk; c++) s = fmaf(q[c], to_f32(k[c]), s);
			if (a.r1) s -= wa_bias(r1, r2, i - j);
		}
		const float mn = fmaxf(m, warp_max(s)), corr = expf(m - mn), p = expf(s - mn);
		l = l * corr + warp_sum(p);
		m = mn;
		for (int c = lane; c < a.dvp; c += 32) o[c] *= corr;
		const int cnt = min(32, total - n0);
		for (int e = 0; e < cnt; e++) {
			const int n2 = n0 + e, j = n2 < kept ? n2 : first + n2 - kept;
			const CT *v = n2 < kept ? vs + size_t(j) * a.G * a.dvp + g * a.dvp : vc + size_t(j % a.cap) * a.G * a.dvp + g * a.dvp;
			const float pe = __shfl_sync(0xffffffffu, p, e);
			for (int c = lane; c < a.dvp; c += 32) o[c] = fmaf(pe, to_f32(v[c]), o[c]);
		}
	}
	PT *out = reinterpret_cast<PT *>(a.out) + size_t(r) * a.ldo + h * a.dvp;
	const float f = a.out_scale / l;
	for (int c = lane; c < a.dvp; c += 32) {
		const float gate = a.p_g >= 0 ? sigmoid_f(to_f32(row[a.p_g + h * a.dvp + c])) : 1.0f;
		out[c] = from_f32<PT>(c < a.dv ? o[c] * f * gate : 0.0f);
	}
}

// ------------------------------------------------------------------ portions, tensor cores
// Warps 0-7: softmax, two threads per query row (32 keys of a tile each; they exchange their maxima through shared
// memory). Warp 8: TMA (Q once, then K and V tiles of 64 keys through one ring). Warp 9: issues the MMAs in the order QK(t+1), PV(t), with S double-buffered in TMEM, so that the softmax of a tile
// runs under the MMAs of its neighbours (and two CTAs share an SM where their tiles fit). P replaces S in TMEM, as the
// bf16 operand of PV; O stays in TMEM and is rescaled there only when a row's running maximum has grown by more than 8
// (powers of two), the sums staying exact for any reference maximum. The distance bias within the window is a table in shared memory
// (lanes of consecutive queries read consecutive words); kept tokens, and windows the table does not reach, evaluate it.
constexpr int WT_THREADS = 320, WT_KEYS = 64, WT_TABLE = 2304;
// D += A B with A in TMEM (row = lane, two bf16 per 32-bit column)
__device__ __forceinline__ void tc_mma_ta(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
	asm volatile(
	    "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
	    "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d_tmem),
	    "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
	    : "memory");
}
// 16 columns of this warp's 32 TMEM lanes, complete on return
__device__ __forceinline__ void wt_ld16(uint32_t taddr, uint32_t (&o)[16]) {
	asm volatile(
	    "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
	    : "=r"(o[0]), "=r"(o[1]), "=r"(o[2]), "=r"(o[3]), "=r"(o[4]), "=r"(o[5]), "=r"(o[6]), "=r"(o[7]), "=r"(o[8]), "=r"(o[9]), "=r"(o[10]), "=r"(o[11]),
	      "=r"(o[12]), "=r"(o[13]), "=r"(o[14]), "=r"(o[15])
	    : "r"(taddr)
	    : "memory");
	asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ float ex2_f(float x) {
	float y;
	asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
	return y;
}
struct WtShape {
	int q_bytes, k_bytes, v_bytes, stage, ns, table, total;  // table: entries of the bias table (0: none)
};
__host__ __device__ inline int wt_chunks(int d) { return (d + 63) / 64; }
__host__ __device__ inline WtShape wt_shape(int dkp, int dvp, int window, bool bias) {
	WtShape s;
	s.q_bytes = wt_chunks(dkp) * 128 * 128;
	s.k_bytes = wt_chunks(dkp) * WT_KEYS * 128;
	s.v_bytes = wt_chunks(dvp) * WT_KEYS * 128;
	s.stage = s.k_bytes > s.v_bytes ? s.k_bytes : s.v_bytes;
	s.ns = 4;  // two CTAs per SM where four stages allow it; fewer stages only where one CTA's shared memory ends
	s.table = bias && window + 256 <= WT_TABLE ? window + 256 : 0;
	while (s.ns > 2 && s.q_bytes + s.ns * s.stage + 4 * s.table + 1024 > 220 * 1024) s.ns--;
	s.total = s.q_bytes + s.ns * s.stage + 4 * s.table + 1024;
	return s;
}
__host__ __device__ inline int wt_tmem_cols(int dvp) { return dvp <= 128 ? 256 : 512; }  // O, then two S (and P) buffers of 64

static __global__ void __launch_bounds__(WT_THREADS, 2) window_attn_tc_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kmap,
                                                                           const __grid_constant__ CUtensorMap vmap, const __grid_constant__ CUtensorMap ksmap,
                                                                           const __grid_constant__ CUtensorMap vsmap, WAttnArgs a) {
	pdl_trigger();
	extern __shared__ uint8_t wt_raw[];
	uint8_t *smem = reinterpret_cast<uint8_t *>((uintptr_t(wt_raw) + 1023) & ~uintptr_t(1023));
	__shared__ uint64_t q_bar, full_bar[4], free_bar[4], s_bar[2], p_bar, pv_bar;
	__shared__ uint32_t tmem_base_s;
	__shared__ int s_fail, s_issued;
	__shared__ float s_max[2][2][128];  // [tile parity][half of the row][row]
	const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const WtShape sh = wt_shape(a.dkp, a.dvp, a.window, a.r1 != nullptr);
	const int ncols = wt_tmem_cols(a.dvp);
	if (tid == 0) {
		mbar_init(&q_bar, 1);
		for (int i = 0; i < 4; i++) {
			mbar_init(&full_bar[i], 1);
			mbar_init(&free_bar[i], 1);
		}
		mbar_init(&s_bar[0], 1);
		mbar_init(&s_bar[1], 1);
		mbar_init(&p_bar, 8);
		mbar_init(&pv_bar, 1);
		s_fail = 0;
		s_issued = 0;
		asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
	}
	if (warp == 9) {
		asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(ncols) : "memory");
		asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem = tmem_base_s;
	const uint32_t s_off = uint32_t(ncols - 128);
	pdl_wait();

	const int seg = blockIdx.z, h = blockIdx.y, g = h / (a.H / a.G);
	const int len = a.d.seg_len[seg], row0 = a.d.seg_row[seg], pos = a.d.seg_pos[seg], seq = a.d.seg_seq[seg];
	// the last query tiles have the most keys: they start first
	const int qt = (len + 127) / 128 - 1 - int(blockIdx.x);
	if (qt >= 0) {
		const int nq = min(128, len - qt * 128), i_lo = pos + qt * 128, i_hi = i_lo + nq - 1;
		// key tiles: of the kept first tokens (those outside the first query's .. last query's window), then of the ring
		const int kept = wa_kept(a, i_hi), nkept = (kept + WT_KEYS - 1) / WT_KEYS;
		const int j_first = wa_first(a, i_lo) / WT_KEYS, nring = i_hi / WT_KEYS - j_first + 1;
		const int ntile = nkept + nring;
		const int kch = wt_chunks(a.dkp), vch = wt_chunks(a.dvp);
		auto stage = [&](int n) { return smem + sh.q_bytes + (n % sh.ns) * sh.stage; };

		if (warp == 8) {
			if (lane == 0) {
				mbar_expect_tx(&q_bar, uint32_t(sh.q_bytes));
				for (int c = 0; c < kch; c++) tma_load_2d(smem + c * 128 * 128, &qmap, a.p_q + h * a.dkp + 64 * c, row0 + qt * 128, &q_bar);
				// load n: K of tile n/2 (even n) or V (odd n)
				for (int n = 0; n < 2 * ntile; n++) {
					const int s = n % sh.ns, use = n / sh.ns, t = n >> 1;
					if (use > 0 && !tc_wait(&free_bar[s], (use - 1) & 1, a.err)) {
						s_fail = 1;
						break;
					}
					const bool isv = n & 1, ks = t < nkept;
					const int y = ks ? seq * a.keep_rows + t * WT_KEYS : seq * a.cap + ((j_first + t - nkept) * WT_KEYS) % a.cap;
					mbar_expect_tx(&full_bar[s], uint32_t(isv ? sh.v_bytes : sh.k_bytes));
					const CUtensorMap *m = isv ? (ks ? &vsmap : &vmap) : (ks ? &ksmap : &kmap);
					for (int c = 0; c < (isv ? vch : kch); c++)
						tma_load_2d(stage(n) + c * WT_KEYS * 128, m, g * (isv ? a.dvp : a.dkp) + 64 * c, y, &full_bar[s]);
					s_issued = n + 1;
				}
			}
		} else if (warp == 9) {
			if (lane == 0) {
				const uint32_t id_s = tc_idesc_bf16(WT_KEYS, 0), id_o = tc_idesc_bf16(a.dvp, 1);
				auto qk = [&](int t) -> bool {
					const int n = 2 * t;
					if (!tc_wait(&full_bar[n % sh.ns], (n / sh.ns) & 1, a.err)) return false;
					tc_fence_after();
					const uint32_t qa = smem_u32(smem), ka = smem_u32(stage(n));
					for (int j = 0; j < a.dkp / 16; j++)
						tc_mma(tmem + s_off + uint32_t((t & 1) * 64), tc_sw128_desc(qa + (j >> 2) * 128 * 128 + (j & 3) * 32, 16, 1024),
						       tc_sw128_desc(ka + (j >> 2) * WT_KEYS * 128 + (j & 3) * 32, 16, 1024), id_s, j > 0 ? 1u : 0u);
					tc_commit(&free_bar[n % sh.ns]);
					tc_commit(&s_bar[t & 1]);
					return true;
				};
				bool ok = tc_wait(&q_bar, 0, a.err) && qk(0);
				for (int t = 0; t < ntile && ok; t++) {
					// S buffer (t+1)&1 was read by the softmax of tile t-1 before it arrived on p_bar for that tile
					if (t + 1 < ntile) ok = qk(t + 1);
					const int n = 2 * t + 1;
					ok = ok && tc_wait(&p_bar, t & 1, a.err) && tc_wait(&full_bar[n % sh.ns], (n / sh.ns) & 1, a.err);
					if (!ok) break;
					tc_fence_after();
					const uint32_t va = smem_u32(stage(n)), pt = tmem + s_off + uint32_t((t & 1) * 64);
					for (int j = 0; j < WT_KEYS / 16; j++)
						tc_mma_ta(tmem, pt + uint32_t(j * 8), tc_sw128_desc(va + j * 2048, WT_KEYS * 128, 1024), id_o, (t > 0 || j > 0) ? 1u : 0u);
					tc_commit(&free_bar[n % sh.ns]);
					tc_commit(&pv_bar);
				}
				if (!ok) s_fail = 1;
			}
		} else {
			const int row = tid & 127, half = tid >> 7, quad = warp & 3;
			const int i = i_lo + row;  // this thread's query (rows past nq compute and are not stored)
			const uint32_t lane_addr = uint32_t(quad * 32) << 16, s_col = s_off + uint32_t(half * 32), p_col = s_off + uint32_t(half * 16);
			const float LOG2E = 1.4426950408889634f;
			const float sc = a.scale * LOG2E;
			const float r1 = a.r1 ? a.r1[h] : 0.0f, r2 = a.r1 ? a.r2[h] : 0.0f;
			// minus the bias (in powers of two) of distance x - 64
			float *tab = reinterpret_cast<float *>(smem + sh.q_bytes + sh.ns * sh.stage);
			if (a.r1)
				for (int x = tid; x < sh.table; x += 256) tab[x] = -r1 * __log2f(1.0f + r2 * float(max(0, x - 64)));
			asm volatile("bar.sync 1, 256;" ::: "memory");
			float m = -INFINITY, l = 0.0f;
			// A wait that runs out leaves the warp "dead": it keeps meeting its partner at the named barriers below, so
			// that nobody waits there for good, and does nothing else.
			bool ok = true;
			auto wait = [&](uint64_t *bar, int parity) {
				return __all_sync(0xffffffffu, !*(volatile int *)&s_fail && tc_wait(bar, uint32_t(parity), a.err)) != 0;
			};
			for (int t = 0; t < ntile; t++) {
				const bool ks = t < nkept;
				const int j0 = (ks ? t * WT_KEYS : (j_first + t - nkept) * WT_KEYS) + half * 32;  // first key of this thread's half
				float r[32];
				float mx = -INFINITY;
				if (ok && !wait(&s_bar[t & 1], (t >> 1) & 1)) ok = false;
				if (ok) {
					tc_fence_after();
					uint32_t ra[32];
					tc_ld32(tmem + lane_addr + s_col + uint32_t((t & 1) * 64), ra);
					asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
					if (!a.r1) {
#pragma unroll
						for (int c = 0; c < 32; c++) r[c] = __uint_as_float(ra[c]) * sc;
					} else if (!ks && sh.table) {
						const float *nb = tab + (i - j0 + 64);
#pragma unroll
						for (int c = 0; c < 32; c++) r[c] = fmaf(__uint_as_float(ra[c]), sc, nb[-c]);
					} else {
#pragma unroll
						for (int c = 0; c < 32; c++) r[c] = fmaf(__uint_as_float(ra[c]), sc, -r1 * __log2f(1.0f + r2 * float(max(0, i - j0 - c))));
					}
					// unless every query of the tile sees every key of it: the ring holds a query's window, the copy the
					// kept tokens before it
					if (ks || j0 + 31 > i_lo || (i_lo + 127) - j0 >= a.window) {
						const int lo = (ks ? 0 : wa_first(a, i)) - j0, hi = (ks ? wa_kept(a, i) - 1 : i) - j0;
#pragma unroll
						for (int c = 0; c < 32; c++) r[c] = (c >= lo && c <= hi) ? r[c] : -INFINITY;
					}
					float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
					for (int c = 0; c < 32; c++) mx4[c & 3] = fmaxf(mx4[c & 3], r[c]);
					mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
				}
				s_max[t & 1][half][row] = mx;
				asm volatile("bar.sync %0, 64;" ::"r"(2 + quad) : "memory");
				mx = fmaxf(mx, s_max[t & 1][half ^ 1][row]);
				// P and O may be touched once PV(t-1) is complete
				if (ok && t > 0 && !wait(&pv_bar, (t - 1) & 1)) ok = false;
				if (!ok) {
					s_fail = 1;
					continue;
				}
				tc_fence_after();
				const bool first = m == -INFINITY;
				const bool grow = mx > m + 8.0f || (first && mx > -INFINITY);
				const float mn = grow ? mx : m;
				const float corr = first ? 0.0f : ex2_f(m - mn);
				if (t > 0 && __any_sync(0xffffffffu, grow && !first)) {  // (the whole warp: TMEM accesses are warp-wide)
					const float f = (grow && !first) ? corr : 1.0f;
					for (int c = 16 * half; c < a.dvp; c += 32) {
						uint32_t o[16];
						wt_ld16(tmem + lane_addr + uint32_t(c), o);
#pragma unroll
						for (int q = 0; q < 16; q++) o[q] = __float_as_uint(__uint_as_float(o[q]) * f);
						asm volatile(
						    "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(tmem + lane_addr + uint32_t(c)),
						    "r"(o[0]), "r"(o[1]), "r"(o[2]), "r"(o[3]), "r"(o[4]), "r"(o[5]), "r"(o[6]), "r"(o[7]), "r"(o[8]), "r"(o[9]), "r"(o[10]), "r"(o[11]),
						    "r"(o[12]), "r"(o[13]), "r"(o[14]), "r"(o[15])
						    : "memory");
					}
					asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
				}
				l *= corr;
				m = mn;
				const float ms = m == -INFINITY ? 0.0f : m;
				uint32_t w[16];
				float l4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
				for (int c = 0; c < 16; c++) {
					const float p0 = ex2_f(r[2 * c] - ms), p1 = ex2_f(r[2 * c + 1] - ms);
					l4[c & 3] += p0 + p1;
					w[c] = pack_bf16(p0, p1);
				}
				l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
				// both halves of a row's S have been read (the exchange above), so P may replace it
				asm volatile(
				    "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(tmem + lane_addr + p_col +
				                                                                                                           uint32_t((t & 1) * 64)),
				    "r"(w[0]), "r"(w[1]), "r"(w[2]), "r"(w[3]), "r"(w[4]), "r"(w[5]), "r"(w[6]), "r"(w[7]), "r"(w[8]), "r"(w[9]), "r"(w[10]), "r"(w[11]), "r"(w[12]),
				    "r"(w[13]), "r"(w[14]), "r"(w[15])
				    : "memory");
				asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
				tc_fence_before();
				__syncwarp();
				if (lane == 0) mbar_arrive(&p_bar);
			}
			// the gate of the first 128 columns is requested before the last products are awaited
			const int rr = row0 + qt * 128 + row;
			const bool gated = a.p_g >= 0 && row < nq;
			const __nv_bfloat16 *gate = reinterpret_cast<const __nv_bfloat16 *>(a.p) + size_t(rr) * a.ldp + a.p_g + h * a.dvp;
			uint4 gv[4][2];
			auto load_gate = [&](int c0) {
#pragma unroll
				for (int e = 0; e < 4; e++) {
					const int c = c0 + 32 * e;
					gv[e][0] = gv[e][1] = make_uint4(0, 0, 0, 0);
					if (gated && c < a.dvp) {
						gv[e][0] = *reinterpret_cast<const uint4 *>(gate + c);
						gv[e][1] = *reinterpret_cast<const uint4 *>(gate + c + 8);
					}
				}
			};
			load_gate(16 * half);
			if (ok) ok = wait(&pv_bar, (ntile - 1) & 1);
			if (!ok) s_fail = 1;
			s_max[ntile & 1][half][row] = l;
			asm volatile("bar.sync %0, 64;" ::"r"(2 + quad) : "memory");
			l += s_max[ntile & 1][half ^ 1][row];
			if (ok) {
				tc_fence_after();
				const float f = a.out_scale / l;
				__nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(a.out) + size_t(rr) * a.ldo + h * a.dvp;
				for (int c0 = 16 * half; c0 < a.dvp; c0 += 128) {
					if (c0 >= 128) load_gate(c0);
#pragma unroll
					for (int e = 0; e < 4; e++) {
						const int c = c0 + 32 * e;
						if (c >= a.dvp) break;
						uint32_t o[16];
						wt_ld16(tmem + lane_addr + uint32_t(c), o);
						if (row < nq) {
							const uint32_t gw[8] = {gv[e][0].x, gv[e][0].y, gv[e][0].z, gv[e][0].w, gv[e][1].x, gv[e][1].y, gv[e][1].z, gv[e][1].w};
							uint32_t w[8];
#pragma unroll
							for (int q = 0; q < 8; q++) {
								float x = __uint_as_float(o[2 * q]) * f, y = __uint_as_float(o[2 * q + 1]) * f;
								if (a.p_g >= 0) {
									x *= __fdividef(1.0f, 1.0f + __expf(-bf16_lo(gw[q])));
									y *= __fdividef(1.0f, 1.0f + __expf(-bf16_hi(gw[q])));
								}
								w[q] = pack_bf16(x, y);
							}
							*reinterpret_cast<uint4 *>(out + c) = make_uint4(w[0], w[1], w[2], w[3]);
							*reinterpret_cast<uint4 *>(out + c + 8) = make_uint4(w[4], w[5], w[6], w[7]);
						}
					}
				}
			}
		}
	}
	tc_fence_before();
	__syncthreads();
	if (s_fail && tid == 0) {
		const int last = *(volatile int *)&s_issued;
		for (int n = max(0, last - sh.ns); n < last; n++) tc_wait(&full_bar[n % sh.ns], (n / sh.ns) & 1, a.err);
	}
	__syncthreads();
	tc_fence_after();
	if (warp == 9) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(ncols));
}

// ------------------------------------------------------------------ one token per sequence
// 256 threads; row r of the step is a segment of length 1 whose key and value are already in the cache (or are put there
// first, rotated, normed and pooled, by the CTA whose run ends with them: `append`). The CTA scores
// its run of keys for up to WK_HEADS query heads of key/value head g at a time, in pieces of WK_KEYS; the CTA that
// arrives last merges the runs, applies the gate and writes the heads' rows.
constexpr int WK_KEYS = 64, WK_HEADS = 4;
__host__ __device__ inline size_t wattn_token_smem(int per, int dkp, int dvp) {
	return (size_t(per) * dkp + size_t(WK_HEADS) * WK_KEYS + size_t(8) * WK_HEADS * (dvp < 256 ? dvp : 256) + 3 * WK_HEADS + 8) * 4;
}
// 16 bytes of a cache row -> floats
__device__ __forceinline__ void wk_unpack(const uint4 &u, float (&f)[8]) {
	f[0] = bf16_lo(u.x); f[1] = bf16_hi(u.x); f[2] = bf16_lo(u.y); f[3] = bf16_hi(u.y);
	f[4] = bf16_lo(u.z); f[5] = bf16_hi(u.z); f[6] = bf16_lo(u.w); f[7] = bf16_hi(u.w);
}
__device__ __forceinline__ void wk_unpack(const uint4 &u, float (&f)[4]) {
	f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
}
template <typename PT, typename CT, typename OT>
__device__ void window_attn_token_cta(const WAttnArgs &a, int r, int g, int split, float *sm) {
	const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
	const int per = a.H / a.G, dkp = a.dkp, dvp = a.dvp;
	constexpr int V4 = 16 / int(sizeof(CT));                 // elements of a 16-byte load
	const int cw = dvp < 32 * V4 ? dvp : 32 * V4;            // value columns of a pass
	float *q = sm, *p = q + per * dkp, *acc = p + WK_HEADS * WK_KEYS, *ml = acc + 8 * WK_HEADS * (dvp < 256 ? dvp : 256), *cr = ml + 2 * WK_HEADS;
	__shared__ int s_last;
	const int seg = a.d.row_seg[r], seq = a.d.seg_seq[seg], i = a.d.seg_pos[seg];
	const PT *row = reinterpret_cast<const PT *>(a.p) + size_t(r) * a.ldp;
	const CT *kc = reinterpret_cast<const CT *>(a.kc) + size_t(seq) * a.cap * a.G * dkp + g * dkp, *vc = reinterpret_cast<const CT *>(a.vc) + size_t(seq) * a.cap * a.G * dvp + g * dvp;
	const CT *ks = reinterpret_cast<const CT *>(a.ks) + size_t(seq) * a.keep_rows * a.G * dkp + g * dkp, *vs = reinterpret_cast<const CT *>(a.vs) + size_t(seq) * a.keep_rows * a.G * dvp + g * dvp;
	const int first = wa_first(a, i), kept = wa_kept(a, i), total = kept + i - first + 1;
	const int pieces = (total + WK_KEYS - 1) / WK_KEYS, share = (pieces + a.nsplit - 1) / a.nsplit;
	const int n_lo = split * share * WK_KEYS, n_hi = min(total, (split + 1) * share * WK_KEYS);
	if (a.rot) {
		const float2 *cs = a.cs + size_t(r) * a.ld_cs;
		for (int x = tid; x < per * dkp; x += 256) q[x] = wa_rotated(a, row + a.p_q + (g * per + x / dkp) * dkp, cs, x % dkp) * a.scale;
	} else {
		for (int x = tid; x < per * dkp; x += 256) q[x] = to_f32(row[a.p_q + g * per * dkp + x]) * a.scale;
	}
	if (a.append && n_lo < total && n_hi == total) {  // (the whole CTA)
		const float2 *cs = a.cs + size_t(r) * a.ld_cs;
		CT *kd = const_cast<CT *>(kc) + size_t(i % a.cap) * a.G * dkp, *vd = const_cast<CT *>(vc) + size_t(i % a.cap) * a.G * dvp;
		const PT *kp = row + a.p_k + g * dkp, *vp = row + a.p_v + g * dvp;
		float f = 1.0f;
		if (a.vnorm) {  // (every warp for itself)
			float s = 0.0f;
			for (int c = lane; c < a.dv; c += 32) s = fmaf(to_f32(vp[c]), to_f32(vp[c]), s);
			f = 1.0f / sqrtf(warp_sum(s) / float(a.dv) + a.eps);
		}
		for (int c = tid; c < dkp; c += 256) kd[c] = from_f32<CT>(wa_rotated(a, kp, cs, c));
		for (int c = tid; c < dvp; c += 256) vd[c] = from_f32<CT>(to_f32(vp[c]) * f);
		__syncthreads();
		if (a.pool && (i + 1) % a.pool == 0) wa_pool_block<CT, 256>(a, seq, g, i / a.pool, tid);
	}
	float *part = a.part + ((size_t(r) * a.G + g) * a.nsplit + split) * per * (dvp + 2);
	// lanes of a value row (a power of two), value rows a warp reads at once
	int lpk = 1;
	while (lpk * V4 < cw) lpk *= 2;
	const int kpw = 32 / lpk, vsub = lane / lpk, vcol = (lane % lpk) * V4;
	for (int h0 = 0; h0 < per; h0 += WK_HEADS) {
		const int nh = min(WK_HEADS, per - h0);
		for (int c0 = 0; c0 < dvp; c0 += cw) {  // (more than one pass only for very wide values: scores are formed again)
			float o[WK_HEADS][V4] = {};
			__syncthreads();
			if (tid < WK_HEADS) {
				ml[2 * tid] = -INFINITY;
				ml[2 * tid + 1] = 0.0f;
			}
			__syncthreads();
			for (int n0 = n_lo; n0 < n_hi; n0 += WK_KEYS) {
				{  // scores: four lanes per key
					const int n = n0 + (tid >> 2), sub = tid & 3;
					const bool on = n < n_hi;
					const int j = on ? (n < kept ? n : first + n - kept) : i;
					const CT *k = (on && n < kept) ? ks + size_t(j) * a.G * dkp : kc + size_t(j % a.cap) * a.G * dkp;
					float s[WK_HEADS] = {};
#pragma unroll 4
					for (int c = sub * V4; c < dkp; c += 4 * V4) {
						float kv[V4];
						wk_unpack(*reinterpret_cast<const uint4 *>(k + c), kv);
#pragma unroll
						for (int y = 0; y < WK_HEADS; y++)
							if (y < nh) {
								const float4 *qh = reinterpret_cast<const float4 *>(q + (h0 + y) * dkp + c);
#pragma unroll
								for (int e = 0; e < V4 / 4; e++) {
									const float4 w = qh[e];
									s[y] = fmaf(w.x, kv[4 * e], fmaf(w.y, kv[4 * e + 1], fmaf(w.z, kv[4 * e + 2], fmaf(w.w, kv[4 * e + 3], s[y]))));
								}
							}
					}
#pragma unroll
					for (int y = 0; y < WK_HEADS; y++) {
						s[y] += __shfl_xor_sync(0xffffffffu, s[y], 1);
						s[y] += __shfl_xor_sync(0xffffffffu, s[y], 2);
					}
					if (sub < nh) {
						float v = sub == 0 ? s[0] : (sub == 1 ? s[1] : (sub == 2 ? s[2] : s[3]));
						const int h = g * per + h0 + sub;
						if (a.r1) v -= wa_bias(a.r1[h], a.r2[h], i - j);
						p[sub * WK_KEYS + (tid >> 2)] = on ? v : -INFINITY;
					}
				}
				__syncthreads();
				if (warp < nh) {  // a warp per head: running maximum, weights, sum
					const float s0 = p[warp * WK_KEYS + lane], s1 = p[warp * WK_KEYS + 32 + lane];
					const float mo = ml[2 * warp], mn = fmaxf(mo, warp_max(fmaxf(s0, s1)));
					const float p0 = expf(s0 - mn), p1 = expf(s1 - mn), sum = warp_sum(p0 + p1), corr = expf(mo - mn);
					p[warp * WK_KEYS + lane] = p0;
					p[warp * WK_KEYS + 32 + lane] = p1;
					if (lane == 0) {
						cr[warp] = corr;
						ml[2 * warp + 1] = ml[2 * warp + 1] * corr + sum;
						ml[2 * warp] = mn;
					}
				}
				__syncthreads();
#pragma unroll
				for (int y = 0; y < WK_HEADS; y++) {
					const float corr = y < nh ? cr[y] : 0.0f;
#pragma unroll
					for (int z = 0; z < V4; z++) o[y][z] *= corr;
				}
				const int c = c0 + vcol;
				if (vcol < cw && c < dvp) {
#pragma unroll 4
					for (int e = warp * kpw + vsub; e < WK_KEYS; e += 8 * kpw) {
						const int n = n0 + e;
						if (n >= n_hi) break;
						const int j = n < kept ? n : first + n - kept;
						const CT *v = n < kept ? vs + size_t(j) * a.G * dvp : vc + size_t(j % a.cap) * a.G * dvp;
						float vv[V4];
						wk_unpack(*reinterpret_cast<const uint4 *>(v + c), vv);
#pragma unroll
						for (int y = 0; y < WK_HEADS; y++)
							if (y < nh) {
								const float pe = p[y * WK_KEYS + e];
#pragma unroll
								for (int z = 0; z < V4; z++) o[y][z] = fmaf(pe, vv[z], o[y][z]);
							}
					}
				}
				__syncthreads();  // (p and cr are written again by the next piece)
			}
			// the warp's value rows meet by shuffles, the warps in shared memory
#pragma unroll
			for (int y = 0; y < WK_HEADS; y++)
#pragma unroll
				for (int z = 0; z < V4; z++) {
					float v = o[y][z];
					for (int d = lpk; d < 32; d *= 2) v += __shfl_xor_sync(0xffffffffu, v, d);
					if (y < nh && vsub == 0 && vcol < cw && c0 + vcol < dvp) acc[(warp * WK_HEADS + y) * cw + vcol + z] = v;
				}
			__syncthreads();
			for (int x = tid; x < nh * cw; x += 256) {
				const int y = x / cw, c = x % cw;
				if (c0 + c >= dvp) continue;
				float v = 0.0f;
#pragma unroll
				for (int w = 0; w < 8; w++) v += acc[(w * WK_HEADS + y) * cw + c];
				part[(h0 + y) * (dvp + 2) + c0 + c] = v;
			}
			if (tid < nh) {
				part[(h0 + tid) * (dvp + 2) + dvp] = ml[2 * tid];
				part[(h0 + tid) * (dvp + 2) + dvp + 1] = ml[2 * tid + 1];
			}
		}
	}
	__threadfence();
	__syncthreads();
	if (a.nsplit > 1) {
		if (tid == 0) {
			const unsigned old = atomicAdd(a.tickets + size_t(r) * a.G + g, 1u);
			s_last = old == unsigned(a.nsplit - 1);
			if (s_last) a.tickets[size_t(r) * a.G + g] = 0;
		}
		__syncthreads();
		if (!s_last) return;
		__threadfence();
	}
	const float *all = a.part + (size_t(r) * a.G + g) * a.nsplit * per * (dvp + 2);
	for (int x = tid; x < per * dvp; x += 256) {
		const int hh = x / dvp, c = x % dvp, h = g * per + hh;
		float m = -INFINITY;
		for (int s = 0; s < a.nsplit; s++) m = fmaxf(m, __ldcg(all + (size_t(s) * per + hh) * (dvp + 2) + dvp));
		float o = 0.0f, l = 0.0f;
		for (int s = 0; s < a.nsplit; s++) {
			const float *ps = all + (size_t(s) * per + hh) * (dvp + 2);
			const float ms = __ldcg(ps + dvp);
			if (ms == -INFINITY) continue;  // a run without keys
			const float w = expf(ms - m);
			o = fmaf(w, __ldcg(ps + c), o);
			l = fmaf(w, __ldcg(ps + dvp + 1), l);
		}
		const float gate = a.p_g >= 0 ? sigmoid_f(to_f32(row[a.p_g + h * dvp + c])) : 1.0f;
		reinterpret_cast<OT *>(a.out)[size_t(r) * a.ldo + h * dvp + c] = from_f32<OT>(c < a.dv ? o / l * gate * a.out_scale : 0.0f);
	}
}

}  // namespace tg
