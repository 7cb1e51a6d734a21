// The family-independent half of libtinygemma_b200: errors and counters, the architecture registry, the life
// cycle of models and states, sampling and the generation loops. What a step computes is behind the virtual
// functions of tg_internal.hpp.
#include <cuda_runtime.h>

#include <algorithm>
#include <atomic>
#include <cmath>
#include <cstring>
#include <map>

#include "json.hpp"
#include "kernels_sampler.cuh"
#include "tg_internal.hpp"

using namespace tg;

// ===================================================================== errors, counters, environment
namespace {
thread_local std::string g_err;
std::atomic<long long> g_launches{0};
std::map<std::string, OpenFn> &registry() {
	static std::map<std::string, OpenFn> r;
	return r;
}
}  // namespace

namespace tg {
thread_local bool g_pdl_scope_off = false;
int g_num_sms = 148;

int fail(int code, const std::string &msg) {
	g_err = msg;
	return code;
}
void count_launch(int n) { g_launches.fetch_add(n, std::memory_order_relaxed); }
long long launches() { return g_launches.load(); }
void set_launches(long long n) { g_launches.store(n); }
int check_launch(const char *what) {
	cudaError_t e = cudaGetLastError();
	if (e != cudaSuccess) return fail(TG_ECUDA, std::string(what) + " launch: " + cudaGetErrorString(e));
	return TG_OK;
}
int env_int(const char *name, int dflt) {
	const char *v = std::getenv(name);
	return v ? std::atoi(v) : dflt;
}
int ensure_device(int device) {
	int n = 0;
	cudaError_t e = cudaGetDeviceCount(&n);
	if (e != cudaSuccess || n == 0) {
		cudaGetLastError();
		return fail(TG_ENODEVICE, "no CUDA device available (this library has no CPU path)");
	}
	if (device < 0 || device >= n) return fail(TG_EINVAL, "device index out of range");
	TG_CUDA(cudaSetDevice(device));
	int sms = 0;
	if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device) == cudaSuccess && sms > 0) g_num_sms = sms;
	return TG_OK;
}
PFN_encodeTiled get_encode_fn() {
	static PFN_encodeTiled fn = nullptr;
	if (!fn) {
		void *p = nullptr;
		cudaDriverEntryPointQueryResult q;
		if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
		    q == cudaDriverEntryPointSuccess)
			fn = reinterpret_cast<PFN_encodeTiled>(p);
	}
	return fn;
}
RegisterArch::RegisterArch(const char *name, OpenFn fn) { registry()[name] = fn; }
}  // namespace tg

// ===================================================================== state, common part
int tg_state::alloc_common() {
	TG_CUDA(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking));
	auto zeroed = [&](auto **p, size_t n) -> int {
		TG_CUDA(cudaMalloc(p, n * 4));
		TG_CUDA(cudaMemsetAsync(*p, 0, n * 4, stream));
		return TG_OK;
	};
	ld_logits = (model->n_vocab + 3) & ~3;
	TG_TRY(zeroed(&logits, size_t(B) * ld_logits));
	TG_TRY(zeroed(&xnorm, size_t(B) * model->hidden_size));
	TG_TRY(zeroed(&step_blk, 4 + size_t(3 + STEP_RANDF) * B));
	err_flag = step_blk;
	tok = step_blk + 4;
	randf_count = tok + B;
	log_count = randf_count + B;
	randf_blk = reinterpret_cast<float *>(log_count + B);
	randf = randf_blk;
	randf_cap = STEP_RANDF;
	randf_in_blk = true;
	TG_CUDA(cudaMallocHost(&host_pin, 64 * 1024));
	host_pos.assign(B, 0);
	use_graph = env_int("TG_USE_GRAPH", 1) != 0;
	return TG_OK;
}

void tg_state::free_common() {
	if (graph) cudaGraphExecDestroy(graph);
	cudaFree(logits);
	cudaFree(xnorm);
	cudaFree(tok_log);
	if (!randf_in_blk) cudaFree(randf);
	cudaFree(step_blk);  // err_flag, tok, randf_count, log_count (and the first randf)
	if (host_pin) cudaFreeHost(host_pin);
	if (stream) cudaStreamDestroy(stream);
}

int tg_state::enqueue_decode_step() {
	// The first step of a state runs eagerly so that lazy module loading and
	// cudaFuncSetAttribute happen outside stream capture; the graph is captured
	// on the second step and replayed from then on.
	if (!use_graph || !warmed) {
		warmed = true;
		return enqueue_decode_all();
	}
	if (!graph) {
		cudaGraph_t g = nullptr;
		const long long before = launches();
		TG_CUDA(cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal));
		int rc = enqueue_decode_all();
		cudaError_t e = cudaStreamEndCapture(stream, &g);
		graph_launches = int(launches() - before);
		set_launches(before);
		if (rc != TG_OK) {
			if (g) cudaGraphDestroy(g);
			return rc;
		}
		if (e != cudaSuccess) return fail(TG_ECUDA, std::string("cudaStreamEndCapture: ") + cudaGetErrorString(e));
		e = cudaGraphInstantiate(&graph, g, 0);
		cudaGraphDestroy(g);
		if (e != cudaSuccess) return fail(TG_ECUDA, std::string("cudaGraphInstantiate: ") + cudaGetErrorString(e));
	}
	TG_CUDA(cudaGraphLaunch(graph, stream));
	count_launch(graph_launches);
	return TG_OK;
}

SampleArgs tg_state::sample_args(float minp, float temp, bool log_tokens) {
	SampleArgs a{};
	a.logits = logits;
	a.V = ld_logits;
	a.tok_out = tok;
	a.tok_log = log_tokens ? tok_log : nullptr;
	a.log_count = log_count;
	a.log_cap = log_cap;
	a.B = B;
	a.minp = minp;
	a.temp = temp;
	a.randf = randf;
	a.randf_count = randf_count;
	a.randf_cap = randf_cap;
	return a;
}

int tg_state::enqueue_sampler(float minp, float temp, bool log_tokens) {
	SampleArgs a = sample_args(minp, temp, log_tokens);
	if (minp < 1.0f) {  // transformer.hpp:208,229: min-p sampling iff minp < 1
		minp_kernel<<<B, SM_THREADS, 0, stream>>>(a);
		count_launch();
		return check_launch("minp");
	}
	launch_k(argmax_kernel, dim3(B), dim3(SM_THREADS), 0, stream, a);
	count_launch();
	return check_launch("argmax");
}

int tg_state::run_steps(int n_steps, float minp, float temp) {
	for (int i = 0; i < n_steps; i++) {
		TG_TRY(enqueue_decode_step());
		TG_TRY(enqueue_sampler(minp, temp, true));
	}
	return TG_OK;
}

int tg_state::step(int, const int *, const int *, const int *, const int *, const int *, float *) {
	return fail(TG_EINVAL, std::string("tg_step: not offered by the family of ") + model->arch());
}
int tg_state::free_sequence(int) {
	return fail(TG_EINVAL, std::string("tg_sequence_free: not offered by the family of ") + model->arch());
}

int tg_state::trace_enable(int) { return fail(TG_EINVAL, std::string("no layer trace for ") + model->arch()); }
int tg_state::trace_read(float *, size_t, int *, int *) { return trace_enable(0); }

// the pinned staging buffer may be overwritten only when no enqueued copy still reads it
int tg_state::staging_acquire() {
	if (staging_busy) {
		TG_CUDA(cudaStreamSynchronize(stream));
		staging_busy = false;
	}
	return TG_OK;
}

// the error word a kernel left (read back by the caller) -> return code; clears the word on the device
int tg_state::report_err(int flag) {
	if (!flag) return TG_OK;
	cudaMemsetAsync(err_flag, 0, 4, stream);
	if (flag == 1) return fail(TG_EINVAL, "token id out of range");
	if (flag == 2) return fail(TG_ESTATE, "cache full (max_pos_global reached)");
	if (flag == 6) return fail(TG_ECUDA, "tensor-core kernel: a pipeline wait ran out");
	return fail(TG_ECUDA, "a kernel reported error " + std::to_string(flag));
}

int tg_state::check_err_flag() {
	TG_CUDA(cudaMemcpyAsync(host_pin + 8192, err_flag, 4, cudaMemcpyDeviceToHost, stream));
	TG_CUDA(cudaStreamSynchronize(stream));
	staging_busy = false;
	return report_err(host_pin[8192]);
}

int tg_state::ensure_log(int steps) {
	if (steps <= log_cap) return TG_OK;
	if (tok_log) cudaFree(tok_log);
	tok_log = nullptr;
	log_cap = 0;
	TG_CUDA(cudaMalloc(&tok_log, size_t(steps) * B * 4));
	log_cap = steps;
	return TG_OK;
}

int tg_state::read_logits(float *logits_host) {
	const size_t row = size_t(model->n_vocab) * 4;
	TG_CUDA(cudaMemcpy2DAsync(logits_host, row, logits, size_t(ld_logits) * 4, row, B, cudaMemcpyDeviceToHost, stream));
	return TG_OK;
}

// ===================================================================== C ABI
extern "C" {

const char *tg_last_error(void) { return g_err.c_str(); }
const char *tg_version(void) { return "tiny-gemma_b200 0.2 (sm_100a)"; }

int tg_device_count(int *count) {
	if (!count) return fail(TG_EINVAL, "count is null");
	int n = 0;
	cudaError_t e = cudaGetDeviceCount(&n);
	if (e != cudaSuccess) {
		cudaGetLastError();
		n = 0;
	}
	*count = n;
	return TG_OK;
}

// ---------------------------------------------------------------- models
int tg_model_open(const char *dir, int device, int dtype, tg_model **out) {
	if (!dir || !out) return fail(TG_EINVAL, "null argument");
	if (dtype != TG_BF16 && dtype != TG_F32) return fail(TG_EINVAL, "dtype must be TG_BF16 or TG_F32");
	json::Value cfg;
	std::string err;
	if (!json::parse_file(std::string(dir) + "/config.json", &cfg, &err)) return fail(TG_EIO, err);
	const json::Value *a = cfg.find("architecture");
	if (!a || a->kind != json::Value::STRING) return fail(TG_EINVAL, "config.json names no architecture");
	auto it = registry().find(a->str);
	if (it == registry().end()) return fail(TG_EINVAL, "unknown architecture: " + a->str);
	return it->second(dir, device, dtype, out);
}

int tg_model_vocab(tg_model *m, int *n_vocab) {
	if (!m || !n_vocab) return fail(TG_EINVAL, "null argument");
	*n_vocab = m->n_vocab;
	return TG_OK;
}

int tg_model_hidden_size(tg_model *m, int *hidden_size) {
	if (!m || !hidden_size) return fail(TG_EINVAL, "null argument");
	*hidden_size = m->hidden_size;
	return TG_OK;
}

int tg_model_free(tg_model *m) {
	if (!m) return TG_OK;
	cudaSetDevice(m->device);
	delete m;
	return TG_OK;
}

// ---------------------------------------------------------------- states
int tg_state_create(tg_model *m, int batch, int max_pos_global, tg_state **out) {
	if (!m || !out || batch < 1 || batch > 2048) return fail(TG_EINVAL, "bad argument (batch must be 1..2048)");
	if (max_pos_global <= 0) max_pos_global = m->n_pos;
	if (max_pos_global > m->n_pos) return fail(TG_EINVAL, "max_pos_global exceeds n_pos");
	TG_CUDA(cudaSetDevice(m->device));
	return m->new_state(batch, max_pos_global, out);
}

int tg_state_free(tg_state *s) {
	if (!s) return TG_OK;
	cudaSetDevice(s->model->device);
	if (s->stream) cudaStreamSynchronize(s->stream);
	delete s;
	return TG_OK;
}

int tg_state_reset(tg_state *s) {
	if (!s) return fail(TG_EINVAL, "null state");
	TG_CUDA(cudaSetDevice(s->model->device));
	TG_TRY(s->reset());
	TG_CUDA(cudaMemsetAsync(s->log_count, 0, 4 * s->B, s->stream));
	TG_CUDA(cudaMemsetAsync(s->randf_count, 0, 4 * s->B, s->stream));
	TG_CUDA(cudaMemsetAsync(s->err_flag, 0, 4, s->stream));
	TG_CUDA(cudaStreamSynchronize(s->stream));
	s->host_pos.assign(s->B, 0);
	return TG_OK;
}

int tg_state_position(tg_state *s, int b, int *position) {
	if (!s || !position || b < 0 || b >= s->B) return fail(TG_EINVAL, "bad argument");
	*position = s->host_pos[b];
	return TG_OK;
}

int tg_state_stream(tg_state *s, void **stream) {
	if (!s || !stream) return fail(TG_EINVAL, "null argument");
	*stream = (void *)s->stream;
	return TG_OK;
}

int tg_prefill(tg_state *s, const int *ids, int S, float *logits_host) {
	if (!s || !ids || S < 1) return fail(TG_EINVAL, "bad argument");
	TG_TRY(s->ready());
	if (S > s->model->n_pos) return fail(TG_EINVAL, "prompt longer than n_pos");
	if (S > s->max_pos_global) return fail(TG_EINVAL, "prompt longer than max_pos_global");
	for (int b = 0; b < s->B; b++)
		if (s->host_pos[b] != 0) return fail(TG_ESTATE, "prefill needs an empty KV cache (decode.hpp:78-79)");
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->prefill(ids, S, logits_host);
}

int tg_step(tg_state *s, int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host) {
	if (!s || n < 1 || !seq || !count || !ids) return fail(TG_EINVAL, "bad argument");
	TG_TRY(s->ready());
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->step(n, seq, count, ids, n_want, want, logits_host);
}

int tg_trace_enable(tg_state *s, int on) {
	if (!s) return fail(TG_EINVAL, "null state");
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->trace_enable(on);
}

int tg_trace_read(tg_state *s, float *x_host, size_t cap_floats, int *runs, int *tokens) {
	if (!s || !runs || !tokens) return fail(TG_EINVAL, "null argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->trace_read(x_host, cap_floats, runs, tokens);
}

int tg_sequence_free(tg_state *s, int b) {
	if (!s || b < 0 || b >= s->B) return fail(TG_EINVAL, "bad argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->free_sequence(b);
}

int tg_decode(tg_state *s, const int *ids, float *logits_host) {
	if (!s) return fail(TG_EINVAL, "null state");
	TG_TRY(s->ready());
	TG_CUDA(cudaSetDevice(s->model->device));
	for (int b = 0; b < s->B; b++)
		if (s->host_pos[b] >= s->max_pos_global) return fail(TG_ESTATE, "global KV cache full (max_pos_global reached)");
	if (ids) {
		for (int b = 0; b < s->B; b++)
			if (ids[b] < 0 || ids[b] >= s->model->n_vocab) return fail(TG_EINVAL, "token id out of range");
		TG_TRY(s->staging_acquire());
		std::memcpy(s->host_pin, ids, 4 * s->B);
		TG_CUDA(cudaMemcpyAsync(s->tok, s->host_pin, 4 * s->B, cudaMemcpyHostToDevice, s->stream));
	}
	TG_TRY(s->enqueue_forward());
	for (int b = 0; b < s->B; b++) s->host_pos[b] += 1;
	s->staging_busy = s->staging_busy || ids != nullptr;  // (an earlier asynchronous call's copy may still be queued)
	if (logits_host) {
		TG_TRY(s->read_logits(logits_host));
		TG_TRY(s->check_err_flag());
	}
	// without a host read-back the call only enqueues: the step runs while the caller prepares the sampler
	// call, and a device-side error (a wait that ran out) is reported by the next call that synchronises
	return TG_OK;
}

int tg_append(tg_state *s, const int *ids, int n, float *logits_host) {
	if (!s || !ids || n < 1) return fail(TG_EINVAL, "bad argument");
	if (s->B != 1) return fail(TG_EINVAL, "tg_append: one sequence per state");
	TG_TRY(s->ready());
	TG_CUDA(cudaSetDevice(s->model->device));
	if (s->host_pos[0] + n > s->max_pos_global) return fail(TG_ESTATE, "global KV cache too small for the appended tokens");
	for (int i = 0; i < n; i++)
		if (ids[i] < 0 || ids[i] >= s->model->n_vocab) return fail(TG_EINVAL, "token id out of range");
	return s->append(ids, n, logits_host);
}

// ---------------------------------------------------------------- sampling and generation
int tg_sample_argmax(tg_state *s, int *toks_host) {
	if (!s) return fail(TG_EINVAL, "null state");
	TG_CUDA(cudaSetDevice(s->model->device));
	TG_TRY(s->enqueue_sampler(2.0f, 1.0f, false));
	TG_CUDA(cudaMemcpyAsync(s->host_pin, s->tok, 4 * s->B, cudaMemcpyDeviceToHost, s->stream));
	TG_TRY(s->check_err_flag());  // synchronises
	if (toks_host) std::memcpy(toks_host, s->host_pin, 4 * s->B);
	return TG_OK;
}

int tg_state_set_randf(tg_state *s, const float *randf_host, int n) {
	if (!s || !randf_host || n < 1) return fail(TG_EINVAL, "bad argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	if (n > s->randf_cap) {
		if (s->randf && !s->randf_in_blk) cudaFree(s->randf);
		s->randf = nullptr;
		s->randf_in_blk = false;
		s->randf_cap = 0;
		TG_CUDA(cudaMalloc(&s->randf, size_t(n) * s->B * 4));
		s->randf_cap = n;
		// captured graphs do not hold this pointer (the sampler is launched outside the graph)
	}
	TG_CUDA(cudaMemcpyAsync(s->randf, randf_host, size_t(n) * s->B * 4, cudaMemcpyHostToDevice, s->stream));
	TG_CUDA(cudaMemsetAsync(s->randf_count, 0, 4 * s->B, s->stream));
	TG_CUDA(cudaStreamSynchronize(s->stream));
	s->randf_valid = std::max(s->randf_valid, n);
	return TG_OK;
}

int tg_sample_minp(tg_state *s, float minp, float temp, const float *randf_host, int *toks_host) {
	if (!s || !randf_host) return fail(TG_EINVAL, "bad argument");
	if (!(minp < 1.0f)) return fail(TG_EINVAL, "minp must be < 1 (the reference uses argmax otherwise, transformer.hpp:208)");
	TG_CUDA(cudaSetDevice(s->model->device));
	if (s->randf_cap >= 1 && size_t(s->B) * 4 <= 4096) {
		// one uniform per sequence, staged through pinned memory: no synchronisation before the launch
		s->randf_valid = std::max(s->randf_valid, 1);
		float *stage = reinterpret_cast<float *>(s->host_pin + 4096);
		std::memcpy(stage, randf_host, size_t(s->B) * 4);
		TG_CUDA(cudaMemcpyAsync(s->randf, stage, size_t(s->B) * 4, cudaMemcpyHostToDevice, s->stream));
		TG_CUDA(cudaMemsetAsync(s->randf_count, 0, 4 * s->B, s->stream));
	} else {
		TG_TRY(tg_state_set_randf(s, randf_host, 1));
	}
	TG_TRY(s->enqueue_sampler(minp, temp, false));
	TG_CUDA(cudaMemcpyAsync(s->host_pin, s->tok, 4 * s->B, cudaMemcpyDeviceToHost, s->stream));
	TG_TRY(s->check_err_flag());  // synchronises
	if (toks_host) std::memcpy(toks_host, s->host_pin, 4 * s->B);
	return TG_OK;
}

int tg_logits_read(tg_state *s, float *logits_host) {
	if (!s || !logits_host) return fail(TG_EINVAL, "null argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	TG_TRY(s->read_logits(logits_host));
	TG_CUDA(cudaStreamSynchronize(s->stream));
	return TG_OK;
}

namespace {
// `counters_zeroed`: the caller's upload has already set log_count (and randf_count) to zero
int generate_async(tg_state *s, int n_steps, float minp, float temp, bool counters_zeroed) {
	TG_TRY(s->ready());
	TG_CUDA(cudaSetDevice(s->model->device));
	for (int b = 0; b < s->B; b++)
		if (s->host_pos[b] + n_steps > s->max_pos_global) return fail(TG_ESTATE, "global KV cache too small for n_steps");
	if (minp < 1.0f && s->randf_valid < n_steps) return fail(TG_ESTATE, "upload uniforms first (tg_state_set_randf)");
	TG_TRY(s->ensure_log(n_steps));
	if (!counters_zeroed) TG_CUDA(cudaMemsetAsync(s->log_count, 0, 4 * s->B, s->stream));
	TG_TRY(s->run_steps(n_steps, minp, temp));
	for (int b = 0; b < s->B; b++) s->host_pos[b] += n_steps;
	return TG_OK;
}
}  // namespace

int tg_generate_async(tg_state *s, int n_steps, float minp, float temp) {
	if (!s || n_steps < 1) return fail(TG_EINVAL, "bad argument");
	return generate_async(s, n_steps, minp, temp, false);
}

int tg_state_tokens(tg_state *s, int n_steps, int *toks_host) {
	if (!s || !toks_host || n_steps < 1 || n_steps > s->log_cap) return fail(TG_EINVAL, "bad argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	TG_CUDA(cudaMemcpyAsync(toks_host, s->tok_log, size_t(n_steps) * s->B * 4, cudaMemcpyDeviceToHost, s->stream));
	TG_TRY(s->check_err_flag());
	return TG_OK;
}

int tg_generate(tg_state *s, const int *first_ids, int n_steps, float minp, float temp, const float *randf_host,
                int *toks_host) {
	if (!s || !first_ids || n_steps < 1) return fail(TG_EINVAL, "bad argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	// Short runs (a step at a time from a host loop) go through the pinned staging buffer with one
	// synchronisation at the end: ids and uniforms in, the launch, tokens out.
	const size_t nbytes = size_t(n_steps) * s->B * 4;
	const bool lean = nbytes <= 16384;
	TG_TRY(s->staging_acquire());
	if (minp < 1.0f && !randf_host) return fail(TG_EINVAL, "min-p sampling needs uniforms");
	if (n_steps == 1 && s->B == 1 && s->lean_step() && env_int("TG_LEAN_STEP", 1)) {
		// One token per call (a host loop around the sampler): the step's inputs — id, uniform, zeroed
		// counters — lie next to each other in the state's step block and go up in ONE copy; the error word
		// and the sampled id lie next to each other too and come back in ONE; the persistent kernel leaves
		// its arena and barrier ready for the next launch. So the call is upload, launch, read-back, wait.
		if (first_ids[0] < 0 || first_ids[0] >= s->model->n_vocab) return fail(TG_EINVAL, "token id out of range");
		int *up = s->host_pin;
		up[0] = first_ids[0];  // tok
		up[1] = 0;             // randf_count
		up[2] = 0;             // log_count
		if (minp < 1.0f) {
			std::memcpy(up + 3, randf_host, 4);
			s->randf_valid = std::max(s->randf_valid, 1);
		}
		TG_CUDA(cudaMemcpyAsync(s->tok, up, minp < 1.0f ? 16 : 12, cudaMemcpyHostToDevice, s->stream));
		s->lean_randf = true;
		const int rc = generate_async(s, 1, minp, temp, true);
		s->lean_randf = false;
		if (rc) return rc;
		int *down = s->host_pin + 8192;
		TG_CUDA(cudaMemcpyAsync(down, s->err_flag, 20, cudaMemcpyDeviceToHost, s->stream));  // err_flag, pad, tok
		TG_CUDA(cudaStreamSynchronize(s->stream));
		s->staging_busy = false;
		TG_TRY(s->report_err(down[0]));
		if (toks_host) toks_host[0] = down[4];
		return TG_OK;
	}
	if (minp < 1.0f) {
		if (lean && s->randf_cap >= n_steps) {
			s->randf_valid = std::max(s->randf_valid, n_steps);
			float *stage = reinterpret_cast<float *>(s->host_pin + 4096);
			std::memcpy(stage, randf_host, nbytes);
			TG_CUDA(cudaMemcpyAsync(s->randf, stage, nbytes, cudaMemcpyHostToDevice, s->stream));
			TG_CUDA(cudaMemsetAsync(s->randf_count, 0, 4 * s->B, s->stream));
		} else {
			TG_TRY(tg_state_set_randf(s, randf_host, n_steps));
		}
	}
	for (int b = 0; b < s->B; b++)
		if (first_ids[b] < 0 || first_ids[b] >= s->model->n_vocab) return fail(TG_EINVAL, "token id out of range");
	std::memcpy(s->host_pin, first_ids, 4 * s->B);
	TG_CUDA(cudaMemcpyAsync(s->tok, s->host_pin, 4 * s->B, cudaMemcpyHostToDevice, s->stream));
	TG_TRY(tg_generate_async(s, n_steps, minp, temp));
	if (toks_host && lean) {
		// (stream order: the ids above were consumed by their copy before this one writes the buffer)
		TG_CUDA(cudaMemcpyAsync(s->host_pin, s->tok_log, nbytes, cudaMemcpyDeviceToHost, s->stream));
		TG_TRY(s->check_err_flag());  // synchronises
		std::memcpy(toks_host, s->host_pin, nbytes);
		return TG_OK;
	}
	if (toks_host) return tg_state_tokens(s, n_steps, toks_host);
	TG_CUDA(cudaStreamSynchronize(s->stream));
	return TG_OK;
}

int tg_hidden_read(tg_state *s, float *hidden_host) {
	if (!s || !hidden_host) return fail(TG_EINVAL, "null argument");
	TG_CUDA(cudaSetDevice(s->model->device));
	TG_CUDA(cudaMemcpyAsync(hidden_host, s->xnorm, size_t(s->B) * s->model->hidden_size * 4, cudaMemcpyDeviceToHost, s->stream));
	TG_CUDA(cudaStreamSynchronize(s->stream));
	return TG_OK;
}

int tg_state_check(tg_state *s) {
	if (!s) return fail(TG_EINVAL, "null state");
	TG_CUDA(cudaSetDevice(s->model->device));
	return s->check_err_flag();
}

// ---------------------------------------------------------------- samplers on host buffers
namespace {
struct DevBuf {
	void *p = nullptr;
	~DevBuf() {
		if (p) cudaFree(p);
	}
	int alloc(size_t n) {
		TG_CUDA(cudaMalloc(&p, n));
		return TG_OK;
	}
};
}  // namespace

int tg_argmax_logits(const float *logits, int n, int *tok) {
	if (!logits || !tok || n < 4 || n % 4) return fail(TG_EINVAL, "bad argument (n must be a multiple of 4)");
	TG_TRY(ensure_device(0));
	DevBuf dl, dt, dc;
	TG_TRY(dl.alloc(size_t(n) * 4));
	TG_TRY(dt.alloc(4));
	TG_TRY(dc.alloc(4));
	TG_CUDA(cudaMemcpy(dl.p, logits, size_t(n) * 4, cudaMemcpyHostToDevice));
	SampleArgs a{};
	a.logits = (float *)dl.p;
	a.V = n;
	a.tok_out = (int *)dt.p;
	a.B = 1;
	argmax_kernel<<<1, SM_THREADS>>>(a);
	count_launch();
	TG_TRY(check_launch("argmax"));
	TG_CUDA(cudaMemcpy(tok, dt.p, 4, cudaMemcpyDeviceToHost));
	return TG_OK;
}

int tg_minp_logits(float *logits, int n, float minp, float temp, float randf, int *tok) {
	if (!logits || !tok || n < MP_CHUNK || n % MP_CHUNK) return fail(TG_EINVAL, "bad argument (n must be a multiple of 8192)");
	TG_TRY(ensure_device(0));
	DevBuf dl, dt, dr, dc;
	TG_TRY(dl.alloc(size_t(n) * 4));
	TG_TRY(dt.alloc(4));
	TG_TRY(dr.alloc(4));
	TG_TRY(dc.alloc(4));
	TG_CUDA(cudaMemcpy(dl.p, logits, size_t(n) * 4, cudaMemcpyHostToDevice));
	TG_CUDA(cudaMemcpy(dr.p, &randf, 4, cudaMemcpyHostToDevice));
	TG_CUDA(cudaMemset(dc.p, 0, 4));
	SampleArgs a{};
	a.logits = (float *)dl.p;
	a.V = n;
	a.tok_out = (int *)dt.p;
	a.B = 1;
	a.minp = minp;
	a.temp = temp;
	a.randf = (const float *)dr.p;
	a.randf_count = (int *)dc.p;
	a.randf_cap = 1;
	minp_kernel<<<1, SM_THREADS>>>(a);
	count_launch();
	TG_TRY(check_launch("minp"));
	TG_CUDA(cudaMemcpy(tok, dt.p, 4, cudaMemcpyDeviceToHost));
	TG_CUDA(cudaMemcpy(logits, dl.p, size_t(n) * 4, cudaMemcpyDeviceToHost));
	return TG_OK;
}

int tg_inverse_cdf(const float *p, int n, float cum0, float randf, int *idx, float *cum_out) {
	if (!p || !idx || n < 1) return fail(TG_EINVAL, "bad argument");
	TG_TRY(ensure_device(0));
	DevBuf dp, di, dc;
	TG_TRY(dp.alloc(size_t(n) * 4));
	TG_TRY(di.alloc(4));
	TG_TRY(dc.alloc(4));
	TG_CUDA(cudaMemcpy(dp.p, p, size_t(n) * 4, cudaMemcpyHostToDevice));
	inverse_cdf_kernel<<<1, SM_THREADS>>>((const float *)dp.p, n, cum0, randf, (int *)di.p, (float *)dc.p);
	count_launch();
	TG_TRY(check_launch("inverse_cdf"));
	TG_CUDA(cudaMemcpy(idx, di.p, 4, cudaMemcpyDeviceToHost));
	if (cum_out) TG_CUDA(cudaMemcpy(cum_out, dc.p, 4, cudaMemcpyDeviceToHost));
	return TG_OK;
}

int tg_launch_count(int reset, long long *count) {
	if (count) *count = launches();
	if (reset) set_launches(0);
	return TG_OK;
}

}  // extern "C"
