// mizerax.cu — the Mizerax family of the model registry (family.h): a decoder described by a config.json whose layers run an attention and a
// mixture of experts SIDE BY SIDE on one layer-normed row, and which runs a stretch of its layers several times with the same weights.
//
//   embedding    token row + learned row of the token's position
//   layer        h = layernorm(x);  x <- x + m (ls1 . attention(h) + ls2 . mixture(h)), m one number for the model, ls1 / ls2 vectors
//   attention    H query heads over G key/value heads; per-head RMS norm of queries and keys with a weight shared by the heads; no rotation; queries
//                at position p times 1 + coef ln(floor((p + 1) / every) + 1); score = scale q.k - 2^(-8 (head + 1) / H) (i - j); the softmax's
//                denominator holds one more 1 (a key of score 0 without a value); one sigmoid gate per head; W_o
//   mixture      softmax over E experts and I identity experts; the `top` largest of score + correction are chosen and weighted by their scores as
//                they are; an expert is W_down (silu(W_gate h) . W_up h), an identity expert returns h; a shared expert runs for every token
//   loop         layers start .. stop - 1 run `times` times, every repetition with a cache of its own, and every repetition begins with
//                x <- W_in [x; x_0], x_0 being the embedded row
//   output       layernorm, logits = embedding table . row
//
// The step function, graph replay of one-token steps, uploads, release and the C entry points are the shared sequence engine's
// (seq_family.cuh), the mixture's kernels in order are seq_moe.cuh's.  Per pass and layer run here:
//     once:          embedding with positions; W_in's right half on the embedded rows (the same addend for every repetition)
//     repetition:    rows product [W_in's left half] + that addend
//     layer:         layer_norm -> rows product [q | k | v | g] -> qkv_post (head norms, query temperature, cache rows) -> swa_attn / swa_tile (slope,
//                    sink, head gate fused) on the side stream, beside router -> experts and [shared gate | up] -> [shared down] on the main one
//                    -> rows product [o].  Passes whose products run on the tensor cores store o plainly and one moe_combine joins the experts, the
//                    shared expert and the attention; short steps join the mixture beside the attention and let o's epilogue add itself.
//
// Cache / state manager: per layer RUN one row of normed keys and one of values per position (the design has no window, and no more positions
// than `max_positions`).  Rows need no clearing: a sequence only reads positions it wrote.
//
// Precision: the residual stream, layer and head norms, temperatures, scores, distance bias, softmax, router, gates and every sum are fp32 in
// both modes.  XALM_PRECISION_BF16 keeps matrices and the key/value cache in bf16 and sends dense products of long passes through the tcgen05
// GEMM (fp16 operands, fp32 accumulation); XALM_PRECISION_F32 widens both and uses the fp32 FMA kernels only.
#include "seq_family.cuh"

#include "seq_moe.cuh"

namespace xalm {
namespace {

using namespace mix;
using namespace seq;

struct Layer { // weights and sizes; what a sequence holds lives in Run
	int H = 0, G = 0, d = 0, dv = 0;
	float scale = 1.f, temp_coef = 0.f;
	int temp_every = 0;
	int off_k = 0, off_v = 0, off_g = 0, n_in = 0; // columns of the stacked input projection
	float *norm = nullptr, *norm_b = nullptr, *q_norm = nullptr, *k_norm = nullptr, *slope = nullptr, *sink = nullptr;
	float *ls1 = nullptr, *ls2 = nullptr; // layer scales times residual_mult
	void *w_in = nullptr, *w_o = nullptr;
	WMat m_in, m_o;
	TcWeight t_in, t_o;
	bool has_moe = false;
	MoeWeights moe;
	long long bytes = 0, expert_bytes = 0; // what one run of the layer reads of its matrices; of that, one expert's share
};

struct Run { // one execution of a layer within a pass: the sequence's cache there
	int layer = 0;
	bool begins = false;               // the first layer of a repetition of the loop
	void *kc = nullptr, *vc = nullptr; // (max_tokens, G * d) normed keys, (max_tokens, G * dv) values
};

struct MizeraxModel : SeqModel {
	int max_positions = 0;
	float residual_mult = 1.f;
	bool loops = false;
	std::vector<Layer> layers;
	std::vector<Run> runs;
	void *positions = nullptr, *w_lx = nullptr, *w_l0 = nullptr; // loop.in's halves: the one on x, the one on the embedded row
	WMat m_lx, m_l0;
	TcWeight t_lx, t_l0;
	float* final_norm_b = nullptr;
	// one pass
	float *x = nullptr, *x2 = nullptr, *x0w = nullptr, *hn = nullptr, *proj = nullptr, *att = nullptr, *ao = nullptr;
	int proj_ld = 4;
	float *part_o = nullptr, *part_ml = nullptr;
	unsigned* tickets = nullptr;
	int part_cap = 0;
	MoeBuffers moe;
};
typedef MizeraxModel Mz;

// ---- config.json ------------------------------------------------------------------------------------------------------------------
int parse_layer(Mz* m, size_t li, const xjson::Value& lv) {
	const int W = m->width;
	const std::string p = "l" + std::to_string(li) + ".", type = lv.at("type").str;
	if (type != "attention") return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has mixer type '%s' (this family runs 'attention')", li, type.c_str());
	const xjson::Value& mx = lv.at("mixer");
	Layer L;
	L.H = geti(mx, "heads");
	L.G = mx.contains("kv_heads") ? geti(mx, "kv_heads") : L.H;
	L.d = geti(mx, "dim");
	L.dv = mx.contains("vdim") ? geti(mx, "vdim") : L.d;
	if (L.H <= 0 || L.G <= 0 || L.H % L.G || L.d <= 0 || L.dv <= 0)
		return set_error(XALM_ERR_INVALID, "config: layer %zu: %d query heads over %d key/value heads of %d and %d", li, L.H, L.G, L.d, L.dv);
	L.scale = mx.contains("scale") ? (float) getf(mx, "scale") : 1.f / sqrtf((float) L.d);
	if (const xjson::Value* qt = object_or_null(mx, "q_temp")) {
		L.temp_coef = (float) getf(*qt, "coef");
		L.temp_every = geti(*qt, "every");
		if (L.temp_every < 1 || (double) L.temp_every != getf(*qt, "every")) return set_error(XALM_ERR_INVALID, "config: layer %zu: q_temp.every must be a positive whole number", li);
	}
	expect(m, p + "norm1", {W}, false);
	expect(m, p + "norm1.b", {W}, false);
	expect(m, p + "mix.q", {L.H * L.d, W}, true);
	expect(m, p + "mix.k", {L.G * L.d, W}, true);
	expect(m, p + "mix.v", {L.G * L.dv, W}, true);
	expect(m, p + "mix.q.norm", {L.d}, false);
	expect(m, p + "mix.k.norm", {L.d}, false);
	expect(m, p + "mix.g", {L.H, W}, true);
	expect(m, p + "mix.o", {W, L.H * L.dv}, true);
	expect(m, p + "ls1", {W}, false);
	if (const xjson::Value* mlp = object_or_null(lv, "mlp")) {
		const std::string kind = mlp->contains("kind") ? mlp->at("kind").str : "moe";
		if (kind != "moe") return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has feed-forward kind '%s' (this family runs 'moe')", li, kind.c_str());
		L.has_moe = true;
		MoeWeights& e = L.moe;
		const xjson::Value& r = mlp->at("router");
		e.ff = geti(mlp->at("expert"), "ff");
		e.E = geti(r, "experts");
		e.identity = r.contains("identity") ? geti(r, "identity") : 0;
		e.top = geti(r, "top");
		if (e.ff <= 0 || e.E <= 0 || e.identity < 0 || e.top <= 0 || e.top > e.E + e.identity)
			return set_error(XALM_ERR_INVALID, "config: layer %zu: %d of %d + %d experts of %d", li, e.top, e.E, e.identity, e.ff);
		moe_expect(m, p + "mlp.", e.E, e.ff, true);
		expect(m, p + "mlp.router", {e.E + e.identity, W}, true);
		expect(m, p + "mlp.correction", {e.E + e.identity}, false);
		if (const xjson::Value* sh = object_or_null(*mlp, "shared")) {
			const int sff = geti(*sh, "ff");
			if (sff <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: shared expert of %d", li, sff);
			moe_expect_shared(m, p + "mlp.shared.", &e, sff, false);
		}
		expect(m, p + "ls2", {W}, false);
	}
	m->layers.push_back(std::move(L));
	return XALM_OK;
}

int parse_config(SeqModel* sm, const char* json) {
	Mz* m = static_cast<Mz*>(sm);
	try {
		const xjson::Value c = xjson::Parser::parse(json, strlen(json));
		m->vocab = geti(c, "vocab");
		m->width = geti(c, "width");
		m->max_positions = geti(c, "max_positions");
		if (m->vocab <= 0 || m->width <= 0 || m->max_positions <= 0) return set_error(XALM_ERR_INVALID, "config: vocab / width / max_positions must be positive");
		m->max_tokens = std::min(m->max_tokens, m->max_positions); // a sequence ends where the position table does
		if (const xjson::Value* nv = object_or_null(c, "norm"); nv && nv->contains("eps")) m->eps = (float) getf(*nv, "eps");
		if (c.contains("residual_mult")) m->residual_mult = (float) getf(c, "residual_mult");
		expect(m, "embed", {m->vocab, m->width}, true);
		expect(m, "pos", {m->max_positions, m->width}, true);
		const xjson::Value& layers = c.at("layers");
		if (layers.kind != xjson::Value::Array || layers.arr.empty()) return set_error(XALM_ERR_INVALID, "config: no layers");
		for (size_t li = 0; li < layers.arr.size(); li++) XALM_TRY(parse_layer(m, li, layers.arr[li]));
		std::vector<LayerRun> order;
		XALM_TRY(layer_order(c, (int) m->layers.size(), &order));
		for (const LayerRun& r : order) {
			Run R;
			R.layer = r.layer;
			R.begins = r.pass > 0; // every pass over the loop begins with loop.in's product
			m->loops = m->loops || R.begins;
			m->runs.push_back(R);
		}
		if (m->loops) expect(m, "loop.in", {m->width, 2 * m->width}, true);
		m->n_layers = (int) m->runs.size(); // what read_state counts: layer runs
		expect(m, "final.norm", {m->width}, false);
		expect(m, "final.norm.b", {m->width}, false);
	} catch (const std::exception& e) {
		return set_error(XALM_ERR_INVALID, "config.json: %s", e.what());
	}
	return XALM_OK;
}

// ---- the kernels of one pass ----------------------------------------------------------------------------------------------------------
// head norms, temperature, cache rows, attention: proj -> att, on the fork's side
int enqueue_attention(Mz* m, const Layer& L, const Run& R, int n, const Fork& fk, int* nl) {
	const bool f32 = m->precision == XALM_PRECISION_F32;
	cudaStream_t s = fk.side();
	XALM_TRY(fk.open());
	QkvPostArgs qa = {};
	qa.proj = m->proj; qa.ld = m->proj_ld; qa.q_off = 0; qa.k_off = L.off_k; qa.v_off = L.off_v;
	qa.H = L.H; qa.G = L.G; qa.d = L.d; qa.dv = L.dv;
	qa.norm_qk = 1; qa.q_norm_w = L.q_norm; qa.k_norm_w = L.k_norm; qa.eps = m->eps;
	qa.temp_every = L.temp_every; qa.temp_coef = L.temp_coef;
	qa.kc = R.kc; qa.vc = R.vc; qa.cache_f32 = f32; qa.keep_first = 0; qa.ring = m->max_tokens;
	qa.step = m->d_step;
	XALM_TRY(launch_qkv_post(qa, n, s));
	(*nl)++;
	SwaArgs sa = {};
	sa.q = m->proj; sa.ldq = m->proj_ld; sa.q_off = 0;
	sa.gate = m->proj; sa.ldg = m->proj_ld; sa.g_off = L.off_g; sa.gate_per_head = 1;
	sa.kc = R.kc; sa.vc = R.vc; sa.ring = m->max_tokens; sa.keep_first = 0;
	sa.H = L.H; sa.G = L.G; sa.d = L.d; sa.dv = L.dv;
	sa.window = 0x7fffffff; sa.scale = L.scale; sa.slope = L.slope; sa.sink = L.sink;
	sa.step = m->d_step; sa.out = m->att;
	sa.n_splits = 0;
	sa.part_o = m->part_o; sa.part_ml = m->part_ml; sa.part_cap = m->part_cap; sa.tickets = m->tickets;
	int launches = 1;
	XALM_TRY(launch_swa(sa, n, f32, s, &launches));
	*nl += launches;
	return fk.mark();
}

// experts and shared expert of m->hn; *ca names everything the join adds
int enqueue_mixture(Mz* m, const Layer& L, int n, MoeCombineArgs* ca, int* nl) {
	MoeRouteArgs ra = {};
	ra.score_kind = MOE_SCORE_SOFTMAX; // the weights are the scores themselves
	RowsEpi eg;
	eg.kind = EPI_GLU; eg.glu_act = GLU_SILU;
	XALM_TRY(moe_experts(m, L.moe, m->moe, m->hn, n, ra, eg, ca, nl));
	ca->scale = L.ls2;
	return XALM_OK;
}

int enqueue_pass(SeqModel* sm, int n, int want, int* nl) {
	Mz* m = static_cast<Mz*>(sm);
	cudaStream_t s = m->stream;
	const int W = m->width;
	const size_t hs = (size_t) m->chunk * W;
	float *x = m->x, *x_next = m->x2; // a repetition's product reads the one and writes the other
	if (m->w_bf16)
		embed_streams_kernel<__nv_bfloat16><<<n, norm_threads(W), 0, s>>>((const __nv_bfloat16*) m->embed, m->d_tokens, W, 1, hs, x, 1.f,
		                                                                  (const __nv_bfloat16*) m->positions, m->d_step);
	else embed_streams_kernel<float><<<n, norm_threads(W), 0, s>>>((const float*) m->embed, m->d_tokens, W, 1, hs, x, 1.f, (const float*) m->positions, m->d_step);
	XALM_SEQ_LAUNCH_CHECK("embed");
	if (m->loops) { // what the embedded row adds at the start of every repetition
		RowsEpi e0;
		e0.kind = EPI_STORE; e0.out = m->x0w; e0.ldo = W;
		XALM_TRY(rows_product(m, x, W, m->w_l0, &m->t_l0, n, W, W, e0, nl));
	}
	for (size_t ri = 0; ri < m->runs.size(); ri++) {
		const Run& R = m->runs[ri];
		const Layer& L = m->layers[(size_t) R.layer];
		if (R.begins) { // x <- W_in [x; x_0]
			RowsEpi el;
			el.kind = EPI_STORE; el.out = x_next; el.ldo = W; el.add = m->x0w; el.lda = W;
			XALM_TRY(rows_product(m, x, W, m->w_lx, &m->t_lx, n, W, W, el, nl));
			std::swap(x, x_next);
		}
		XALM_TRY(launch_layer_norm(x, W, L.norm, L.norm_b, m->eps, W, m->hn, n, s));
		(*nl)++;
		RowsEpi est;
		est.kind = EPI_STORE; est.out = m->proj; est.ldo = m->proj_ld;
		XALM_TRY(rows_product(m, m->hn, W, L.w_in, &L.t_in, n, L.n_in, W, est, nl));
		const Fork fk = {m, L.has_moe && tune("seq_overlap") != 0};
		XALM_TRY(enqueue_attention(m, L, R, n, fk, nl));
		MoeCombineArgs ca = {};
		ca.x_in = x; ca.x_out = x;
		if (L.has_moe) XALM_TRY(enqueue_mixture(m, L, n, &ca, nl));
		// Tensor-core passes: the GEMM stores o's product itself and one kernel joins everything.  Short steps: the mixture joins x while the attention
		// still runs, and o's epilogue adds the rest.
		const bool joined = L.has_moe && m->use_tc && L.t_o.hi && n >= m->tc_min_rows;
		if (L.has_moe && !joined) {
			XALM_TRY(launch_moe_combine(ca, n, s));
			(*nl)++;
		}
		XALM_TRY(fk.join());
		RowsEpi eo;
		if (joined) { eo.kind = EPI_STORE; eo.out = m->ao; eo.ldo = W; }
		else { eo.kind = EPI_HC; eo.xs = x; eo.S = 1; eo.stream_stride = hs; eo.scale = L.ls1; }
		XALM_TRY(rows_product(m, m->att, L.H * L.dv, L.w_o, &L.t_o, n, W, L.H * L.dv, eo, nl));
		if (joined) {
			ca.other = m->ao; ca.other_scale = L.ls1;
			XALM_TRY(launch_moe_combine(ca, n, s));
			(*nl)++;
		}
		if (m->keep_layers) XALM_CUDA_CHECK(cudaMemcpyAsync(m->layer_sums + ri * hs, x, (size_t) n * W * 4, cudaMemcpyDeviceToDevice, s));
	}
	if (want) {
		const int rows = want == 2 ? n : 1, first = want == 2 ? 0 : n - 1;
		XALM_TRY(launch_layer_norm(x + (size_t) first * W, W, m->final_norm, m->final_norm_b, m->eps, W, m->hn, rows, s));
		(*nl)++;
		RowsEpi eh;
		eh.kind = EPI_STORE; eh.out = m->logits; eh.ldo = m->vocab;
		XALM_TRY(rows_product(m, m->hn, W, m->w_head, &m->t_head, rows, m->vocab, W, eh, nl));
	}
	return XALM_OK;
}

// ---- device layouts, cache, pass buffers ---------------------------------------------------------------------------------------------
int upload_scaled(SeqModel* m, const std::string& name, float by, float** dst) {
	std::vector<float> v = m->tensors.at(name).v;
	for (float& x : v) x *= by;
	return upload_floats(m, v.data(), v.size(), dst);
}

int finalize(SeqModel* sm) {
	Mz* m = static_cast<Mz*>(sm);
	const int W = m->width;
	const size_t C = (size_t) m->chunk, kelem = m->precision == XALM_PRECISION_F32 ? 4 : 2;
	auto T = [&](const std::string& n) { return tensor_or_null(m, n); };
	size_t max_in = 4, max_att = 1, max_h = 1;
	XALM_TRY(upload_rows(m, {T("pos")}, W, false, &m->positions, nullptr));
	XALM_TRY(upload_vec(m, "final.norm.b", &m->final_norm_b));
	if (m->loops) { // loop.in's columns: the left half reads x, the right half the embedded row
		const HostTensor* both = T("loop.in");
		HostTensor half[2];
		for (int k = 0; k < 2; k++) {
			half[k].shape = {W, W};
			half[k].v.resize((size_t) W * W);
			for (int r = 0; r < W; r++) memcpy(&half[k].v[(size_t) r * W], &both->v[(size_t) r * 2 * W + (size_t) k * W], (size_t) W * 4);
		}
		XALM_TRY(upload_rows(m, {&half[0]}, W, false, &m->w_lx, &m->m_lx));
		XALM_TRY(upload_rows(m, {&half[1]}, W, false, &m->w_l0, &m->m_l0));
	}
	for (size_t li = 0; li < m->layers.size(); li++) {
		Layer& L = m->layers[li];
		const std::string p = "l" + std::to_string(li) + ".";
		const int H = L.H, G = L.G, d = L.d, dv = L.dv;
		const long long bytes0 = m->weight_bytes;
		XALM_TRY(upload_vec(m, p + "norm1", &L.norm));
		XALM_TRY(upload_vec(m, p + "norm1.b", &L.norm_b));
		XALM_TRY(upload_vec(m, p + "mix.q.norm", &L.q_norm));
		XALM_TRY(upload_vec(m, p + "mix.k.norm", &L.k_norm));
		XALM_TRY(upload_scaled(m, p + "ls1", m->residual_mult, &L.ls1));
		L.off_k = H * d; L.off_v = L.off_k + G * d; L.off_g = L.off_v + G * dv;
		L.n_in = (L.off_g + H + 3) / 4 * 4; // rows of zeros round the stack up to what the tensor-core GEMM takes
		HostTensor zeros;
		zeros.shape = {L.n_in - L.off_g - H, W};
		zeros.v.assign((size_t) zeros.shape[0] * W, 0.f);
		XALM_TRY(upload_rows(m, {T(p + "mix.q"), T(p + "mix.k"), T(p + "mix.v"), T(p + "mix.g"), &zeros}, W, false, &L.w_in, &L.m_in));
		XALM_TRY(upload_rows(m, {T(p + "mix.o")}, H * dv, false, &L.w_o, &L.m_o));
		std::vector<float> slope((size_t) H);
		for (int h = 0; h < H; h++) slope[(size_t) h] = (float) exp2(-8.0 * (h + 1) / H);
		XALM_TRY(upload_floats(m, slope.data(), slope.size(), &L.slope));
		XALM_TRY(dev_alloc(m, &L.sink, (size_t) H, true)); // every head's sink scores 0
		if (!swa_pick_tq(H, G, d, dv, m->chunk) && swa_smem_bytes(H, d, dv) > 200 * 1024)
			return set_error(XALM_ERR_UNSUPPORTED, "layer %zu: attention heads need %zu bytes of shared memory", li, swa_smem_bytes(H, d, dv));
		XALM_TRY(swa_prepare(H, d, dv));
		if (L.has_moe) {
			XALM_TRY(upload_scaled(m, p + "ls2", m->residual_mult, &L.ls2));
			XALM_TRY(upload_vec(m, p + "mlp.correction", &L.moe.correction));
			XALM_TRY(moe_upload(m, p + "mlp.", true, &L.moe, &m->moe));
			L.expert_bytes = 3ll * L.moe.ff * W * (m->w_bf16 ? 2 : 4);
		}
		L.bytes = m->weight_bytes - bytes0;
		max_in = std::max(max_in, (size_t) L.n_in);
		max_att = std::max(max_att, (size_t) H * dv);
		max_h = std::max(max_h, (size_t) H);
	}
	XALM_TRY(layer_norm_prepare(W));
	if (m->loops) {
		XALM_TRY(tc_register(m, m->m_lx, &m->t_lx));
		XALM_TRY(tc_register(m, m->m_l0, &m->t_l0));
	}
	for (Layer& L : m->layers) {
		XALM_TRY(tc_register(m, L.m_in, &L.t_in));
		XALM_TRY(tc_register(m, L.m_o, &L.t_o));
		if (L.has_moe) XALM_TRY(moe_tc_register(m, &L.moe, &m->moe));
	}
	// what the sequence holds, per layer run
	for (Run& R : m->runs) {
		const Layer& L = m->layers[(size_t) R.layer];
		uint8_t *kc = nullptr, *vc = nullptr;
		XALM_TRY(dev_alloc(m, &kc, (size_t) m->max_tokens * L.G * L.d * kelem, true));
		XALM_TRY(dev_alloc(m, &vc, (size_t) m->max_tokens * L.G * L.dv * kelem, true));
		R.kc = kc; R.vc = vc;
	}
	m->proj_ld = (int) ((max_in + 3) / 4 * 4);
	m->part_cap = std::max(4 * 64, 4 * m->chunk); // one-token steps: up to 64 key splits; passes of a prompt: up to 4 per token
	XALM_TRY(dev_alloc(m, &m->x, C * W));
	XALM_TRY(dev_alloc(m, &m->x2, C * W));
	XALM_TRY(dev_alloc(m, &m->x0w, C * W));
	XALM_TRY(dev_alloc(m, &m->hn, C * W));
	XALM_TRY(dev_alloc(m, &m->proj, C * m->proj_ld));
	XALM_TRY(dev_alloc(m, &m->att, C * max_att));
	XALM_TRY(dev_alloc(m, &m->ao, C * W));
	XALM_TRY(dev_alloc(m, &m->part_o, (size_t) m->part_cap * max_att));
	XALM_TRY(dev_alloc(m, &m->part_ml, (size_t) m->part_cap * 2 * max_h));
	XALM_TRY(dev_alloc(m, &m->tickets, 8 * C, true));
	return moe_alloc(m, &m->moe);
}

int release(SeqModel*) { return XALM_OK; } // nothing but cache rows, and a sequence only reads positions it wrote

// beyond one reading of every matrix: repeated layers (and loop.in's left half) read theirs again, a mixture reads only the chosen experts; the
// visible cache rows
long long active_bytes(SeqModel* sm, long long pos) {
	Mz* m = static_cast<Mz*>(sm);
	const long long W = m->width, kelem = m->precision == XALM_PRECISION_F32 ? 4 : 2, welem = m->w_bf16 ? 2 : 4;
	// the embedding table is read once more, whole, as the head matrix; of the position table one row
	long long b = (m->vocab - 1) * W * welem - (m->max_positions - 1) * W * welem;
	std::vector<int> seen(m->layers.size(), 0);
	int passes = 0;
	for (const Run& R : m->runs) {
		const Layer& L = m->layers[(size_t) R.layer];
		const int skipped = L.has_moe ? std::max(0, L.moe.E - L.moe.top) : 0;
		const long long live = L.bytes - skipped * L.expert_bytes;
		b += seen[(size_t) R.layer]++ ? live : live - L.bytes;
		b += (pos + 1) * L.G * (L.d + L.dv) * kelem;
		passes += R.begins;
	}
	return b + std::max(0, passes - 1) * W * W * welem;
}

bool state_buffer(SeqModel*, int, const float**, size_t*) { return false; }

void destroy(SeqModel* sm) {
	Mz* m = static_cast<Mz*>(sm);
	tc_weight_free(&m->t_lx);
	tc_weight_free(&m->t_l0);
	for (Layer& L : m->layers) {
		for (TcWeight* t : {&L.t_in, &L.t_o}) tc_weight_free(t);
		moe_free(&L.moe);
	}
	delete m;
}

const SeqHooks mizerax_hooks = {parse_config, finalize, enqueue_pass, release, active_bytes, state_buffer, destroy};
extern const ModelFamily mizerax_family;
int create(const char* json, int device, int max_tokens, int precision, xalm_cuda_model** out) {
	return seq_create<Mz>(&mizerax_family, &mizerax_hooks, json, device, max_tokens, precision, out);
}
const ModelFamily mizerax_family = seq_family_table("Mizerax", create);
const FamilyRegistrar mizerax_registrar(&mizerax_family);

} // namespace
} // namespace xalm
