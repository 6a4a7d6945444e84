// bolapel.cu -- the Bolapel architecture (arch.h): a decoder with an RMS norm before and after every sublayer,
//     x <- x + rms(mixer(shift(rms(x) n1))) n1b;      x <- x + rms(ff(rms(x) n2)) n2b       (a layer may have no ff)
// shift(h)_t = h_t + (h_{t-1} - h_t) * mu per channel (h_{-1} = 0): the previous token's normed row is a layer's state.  Two kinds of
// sequence mixer, listed per layer in config.json "layers":
//   "general_delta"  generalized delta rule: r, k, v = W h, decay per head and key channel w = exp(-e^{-1/2} sigmoid(W_2 tanh(W_1 h) +
//                    w0)), removal rate a = sigmoid(W_a h + b), unit key u:  S <- diag(w) S - (a u)(u^T S) + k v^T,  o = S^T r;
//                    o RMS-normed per head, all heads times one weight row and sigmoid(W_g h)
//   "attention"      grouped heads, q and k RMS-normed per head with a weight, the first rot.dims dimensions turned (i with
//                    i + dims/2), keys of the same block of mask.size positions only, weights sigmoid(score + bias of the head)
//                    that are not normalised, one sigmoid gate per head; a layer with "kv_from" reads the cache of that layer
// and a dense SiLU GLU.  logits = cap tanh(head(rms(x) w) / cap).  Everything model-specific comes from config.json and the tensor
// shapes; the kernels are the generic ones of dense_ops.cuh / mixer_ops.cuh / dense_gemm.cuh, the step / chunking / graph machinery
// is DenseModel's.  Caches are addressed by position like those of the other models; recurrent states and shift rows continue from
// the previous step and restart when a step begins at position 0.
#include "dense_model.cuh"
#include "mixer_ops.cuh"

namespace lmrs {
namespace {

enum BoMixer { BO_DELTA = 0, BO_ATTENTION = 1 };

struct BoLayerCfg {
    int kind = BO_DELTA;
    int H = 0, d = 0, ra = 0;                    // delta rule
    int G = 0, dk = 0, dv = 0;                   // attention
    float scale = 1.0f;
    int chunk = 0, rot_dims = 0, kv_from = -1;
    double rot_base = 10000.0;
    int ff = 0;                                  // 0: no feed-forward
};

template <typename AT, typename WT> class BolapelModel : public DenseModel<AT, WT> {
  public:
    typedef DenseModel<AT, WT> B;
    using B::load_vec; using B::load_stack; using B::error; using B::launches; using B::info; using B::d_logits; using B::width; using B::vocab;
    using B::max_tokens; using B::sms; using B::d_tokens; using B::cap; using B::x; using B::hn; using B::d_rows; using B::MAX_SPLIT; using B::pdl_now;
    using B::dalloc; using B::dfree; using B::need; using B::upload_w; using B::check_launch; using B::launch_k; using B::drop_graphs; using B::optin;

    struct Layer {
        BoLayerCfg c;
        float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *mu = nullptr;
        float* prev = nullptr;                   // [2][width]: the last token's normed row; second half: where a many-row step leaves the new one
        WT* w_in = nullptr; int in_rows = 0;     // fused input projection of the mixer (rows padded to a multiple of 8)
        WT* wo = nullptr; int wo_cols = 0;
        // delta rule
        WT* w2 = nullptr;
        float *w0 = nullptr, *a_bias = nullptr, *onorm = nullptr, *state = nullptr;
        // attention
        float *qnorm = nullptr, *knorm = nullptr, *wbias = nullptr, *kcache = nullptr, *vcache = nullptr;   // caches: the lender's when kv_from
        const float *rot_cos = nullptr, *rot_sin = nullptr;
        // feed-forward
        WT *wgate = nullptr, *wup = nullptr, *wdown = nullptr;
    };
    std::vector<Layer> layers;
    WT *embed = nullptr, *head = nullptr;
    float* final_norm = nullptr;
    float softcap = 0.0f, decay_rate = (float)exp(-0.5);
    float* shift_rows = nullptr;   // [2][layers][width]
    uint32_t next_pos = 0;         // where the recurrent states and shift rows stand
    // scratch for `cap` rows
    float *proj = nullptr, *qa = nullptr, *gate = nullptr, *z = nullptr, *rec = nullptr, *fo = nullptr, *yf = nullptr, *part = nullptr, *inv = nullptr;
    AT *h = nullptr, *lat = nullptr, *att = nullptr, *act = nullptr;
    int max_proj = 0, max_ra = 0, max_q = 0, max_n = 0, max_H = 0, max_dv = 0, max_att = 0, max_ff = 0;
    // test / measurement overrides: another thread layout of the scan; one-token steps through the many-token kernels
    int scan_shape = 0, step_fused = 1;

    size_t n_layers() const override { return layers.size(); }

    // ---- configuration ---------------------------------------------------------------------------------------------------
    int parse_layer(const Json& jl, size_t li, BoLayerCfg& c) {
        const std::string type = jl.at("type").str, where = "config.json layers[" + std::to_string(li) + "]";
        const Json& m = jl.at("mixer");
        if (type == "general_delta") {
            c.kind = BO_DELTA;
            c.H = (int)m.at("heads").number(0); c.d = (int)m.at("dim").number(0);
            if (c.H <= 0 || c.d <= 0) { error = where + ": bad head geometry"; return 1; }
            if (c.d > DELTA_MAX_DK) { error = where + ": dim above " + std::to_string(DELTA_MAX_DK) + " is not supported by the delta-rule kernel"; return 1; }
        } else if (type == "attention") {
            c.kind = BO_ATTENTION;
            c.H = (int)m.at("heads").number(0); c.G = (int)m.at("kv_heads").number(c.H);
            c.dk = (int)m.at("dim").number(0); c.dv = (int)m.at("vdim").number(c.dk);
            c.scale = (float)m.at("scale").number(1.0);
            c.chunk = m.has("mask") ? (int)m.at("mask").at("size").number(0) : 0;
            if (m.has("rot")) { c.rot_dims = (int)m.at("rot").at("dims").number(0); c.rot_base = m.at("rot").at("base").number(10000.0); }
            if (m.has("kv_from")) c.kv_from = (int)m.at("kv_from").number(-1);
            if (c.H <= 0 || c.G <= 0 || c.dk <= 0 || c.dv <= 0 || c.H % c.G != 0) { error = where + ": bad head geometry"; return 1; }
            if (c.chunk < 0) { error = where + ": mask.size must not be negative"; return 1; }
            if (c.rot_dims < 0 || c.rot_dims > c.dk || c.rot_dims % 2 != 0) { error = where + ": rot.dims must be even and at most dim"; return 1; }
            if (!B::attention_fits(c.dk, c.dv)) { error = where + ": head dim " + std::to_string(c.dk) + " / vdim " + std::to_string(c.dv) + " do not fit the attention kernel's shared-memory tiles"; return 1; }
            if (m.has("kv_from")) {
                if (c.kv_from < 0 || c.kv_from >= (int)li) { error = where + ": kv_from must name an earlier layer"; return 1; }
                const BoLayerCfg& l = layers[c.kv_from].c;
                if (l.kind != BO_ATTENTION || l.kv_from >= 0 || l.G != c.G || l.dk != c.dk || l.dv != c.dv) {
                    error = where + ": kv_from must name an attention layer with keys and values of its own and the same key/value heads";
                    return 1;
                }
            }
        } else { error = where + ": unknown layer type '" + type + "'"; return 1; }
        if (jl.has("mlp")) {
            const Json& f = jl.at("mlp");
            if (f.has("kind") && f.at("kind").str != "dense") { error = where + ": unknown mlp kind '" + f.at("kind").str + "'"; return 1; }
            c.ff = (int)f.at("ff").number(0);
            if (c.ff <= 0) { error = where + ": mlp.ff is required"; return 1; }
        }
        return 0;
    }

    // ---- weights -----------------------------------------------------------------------------------------------------------
    int load_delta(const SafeTensors& st, const std::string& q, Layer& L) {
        BoLayerCfg& c = L.c;
        const int n = c.H * c.d;
        const StTensor* t = st.find(q + "w1");
        if (!t || t->shape.size() != 2) { error = "tensor '" + q + "w1' is missing"; return 1; }
        c.ra = (int)t->shape[0];
        if (load_stack(st, {{q + "r", n}, {q + "k", n}, {q + "v", n}, {q + "g", n}, {q + "a", n}, {q + "w1", c.ra}}, width, &L.w_in, &L.in_rows, 8) ||
            load_stack(st, {{q + "w2", n}}, c.ra, &L.w2, nullptr) || load_stack(st, {{q + "o", width}}, n, &L.wo, nullptr) ||
            load_vec(st, q + "w0", n, &L.w0) || load_vec(st, q + "a.b", n, &L.a_bias) || load_vec(st, q + "norm", n, &L.onorm))
            return 1;
        const size_t ns = (size_t)n * c.d;
        if (dalloc(&L.state, ns)) return 1;
        GCK(cudaMemset(L.state, 0, ns * 4));
        L.wo_cols = n;
        max_ra = std::max(max_ra, c.ra);
        max_n = std::max(max_n, n);
        return 0;
    }
    int load_attention(const SafeTensors& st, const std::string& q, Layer& L) {
        BoLayerCfg& c = L.c;
        const int nq = c.H * c.dk, nk = c.G * c.dk, nv = c.G * c.dv;
        if (c.kv_from >= 0) {
            if (load_stack(st, {{q + "q", nq}, {q + "g", c.H}}, width, &L.w_in, &L.in_rows, 8)) return 1;
            L.kcache = layers[c.kv_from].kcache; L.vcache = layers[c.kv_from].vcache;
        } else {
            if (load_stack(st, {{q + "q", nq}, {q + "k", nk}, {q + "v", nv}, {q + "g", c.H}}, width, &L.w_in, &L.in_rows, 8) ||
                load_vec(st, q + "k.norm", c.dk, &L.knorm) || dalloc(&L.kcache, (size_t)max_tokens * nk) || dalloc(&L.vcache, (size_t)max_tokens * nv))
                return 1;
        }
        if (load_vec(st, q + "q.norm", c.dk, &L.qnorm) || load_vec(st, q + "pb", c.H, &L.wbias)) return 1;
        L.wo_cols = c.H * c.dv;
        if (load_stack(st, {{q + "o", width}}, L.wo_cols, &L.wo, nullptr)) return 1;
        if (c.rot_dims > 0) {
            std::vector<double> f;
            for (int i = 0; i < c.rot_dims / 2; i++) f.push_back(pow(c.rot_base, -2.0 * (double)i / (double)c.rot_dims));
            char key[160];
            snprintf(key, sizeof key, "plain/%d/%.17g", c.rot_dims, c.rot_base);
            if (this->angle_tables(key, f, 1.0, &L.rot_cos, &L.rot_sin)) return 1;
        }
        max_q = std::max(max_q, nq);
        max_H = std::max(max_H, c.H);
        max_dv = std::max(max_dv, c.dv);
        return 0;
    }

    int load(const std::string& dir, const Json& cfg, const ArchOptions& opt) {
        sms = opt.sms;
        B::gemm_ctx.sms = opt.sms;
        width = (int)cfg.at("width").number(0);
        vocab = (int)cfg.at("vocab").number(0);
        if (width <= 0 || vocab <= 0) { error = "config.json: width and vocab are required"; return 1; }
        const float eps = (float)cfg.at("norm").at("eps").number(1e-6);
        softcap = cfg.has("logit_softcap") ? (float)cfg.at("logit_softcap").number(0.0) : 0.0f;
        max_tokens = opt.max_tokens ? opt.max_tokens : 4096u;
        const Json& jl = cfg.at("layers");
        if (jl.kind != Json::ARR || jl.arr.empty()) { error = "config.json: 'layers' must be a non-empty list"; return 1; }
        SafeTensors st;
        if (!st.open(dir + "/model.safetensors", error)) return 1;
        if (load_stack(st, {{"embed", vocab}}, width, &embed, nullptr) || load_stack(st, {{"head", vocab}}, width, &head, nullptr) ||
            load_vec(st, "final.norm", width, &final_norm))
            return 1;
        layers.resize(jl.arr.size());
        const size_t nl = layers.size();
        if (dalloc(&shift_rows, 2 * nl * width)) return 1;
        GCK(cudaMemset(shift_rows, 0, 2 * nl * width * 4));
        for (size_t li = 0; li < nl; li++) {
            Layer& L = layers[li];
            if (parse_layer(jl.arr[li], li, L.c)) return 1;
            const std::string p = "l" + std::to_string(li) + ".";
            L.prev = shift_rows + li * width;
            if (load_vec(st, p + "norm1", width, &L.norm1) || load_vec(st, p + "norm1b", width, &L.norm1b) || load_vec(st, p + "shift", width, &L.mu)) return 1;
            if (L.c.kind == BO_DELTA ? load_delta(st, p + "mix.", L) : load_attention(st, p + "mix.", L)) return 1;
            max_proj = std::max(max_proj, L.in_rows);
            max_att = std::max(max_att, L.wo_cols);
            if (L.c.ff > 0) {
                if (load_vec(st, p + "norm2", width, &L.norm2) || load_vec(st, p + "norm2b", width, &L.norm2b) ||
                    load_stack(st, {{p + "mlp.gate", L.c.ff}}, width, &L.wgate, nullptr) || load_stack(st, {{p + "mlp.up", L.c.ff}}, width, &L.wup, nullptr) ||
                    load_stack(st, {{p + "mlp.down", width}}, L.c.ff, &L.wdown, nullptr))
                    return 1;
                max_ff = std::max(max_ff, L.c.ff);
            }
        }
        if (dalloc(&d_tokens, (size_t)max_tokens) || dalloc(&d_logits, (size_t)vocab)) return 1;
        GCK(cudaMemset(d_tokens, 0, (size_t)max_tokens * 4));
        const BoLayerCfg& c0 = layers[0].c;
        info.architecture = "Bolapel";
        info.model_type = 7;
        info.vocab = (uint32_t)vocab; info.width = (uint32_t)width; info.n_layers = (uint32_t)nl; info.max_tokens = max_tokens;
        info.heads = (uint32_t)c0.H; info.kv_heads = (uint32_t)(c0.kind == BO_DELTA ? c0.H : c0.G); info.head_dim = (uint32_t)(c0.kind == BO_DELTA ? c0.d : c0.dk);
        info.ff = (uint32_t)c0.ff; info.dtype = opt.dtype; info.eps = eps;
        return ensure_scratch(1);
    }

    int ensure_scratch(size_t rows) override {
        if (rows <= cap) return 0;
        drop_graphs();   // captured launches point into the old scratch
        for (void* p : {(void*)x, (void*)hn, (void*)d_rows, (void*)h, (void*)lat, (void*)att, (void*)act, (void*)proj, (void*)qa, (void*)gate, (void*)z,
                        (void*)rec, (void*)fo, (void*)yf, (void*)part, (void*)inv})
            dfree(p);
        x = nullptr; hn = nullptr; d_rows = nullptr; h = nullptr; lat = nullptr; att = nullptr; act = nullptr; proj = nullptr; qa = nullptr; gate = nullptr;
        z = nullptr; rec = nullptr; fo = nullptr; yf = nullptr; part = nullptr; inv = nullptr;
        cap = 0;
        int max_heads = 1;
        size_t max_rec = 0;   // floats of a four-token block's records
        for (const Layer& L : layers) {
            max_heads = std::max(max_heads, L.c.H);
            if (L.c.kind == BO_DELTA) max_rec = std::max(max_rec, (size_t)L.c.H * gd_record(scan_rows(L.c.d)));
        }
        if (dalloc(&x, rows * width) || dalloc(&hn, rows * width) || dalloc(&d_rows, rows) || dalloc(&h, rows * width) || dalloc(&lat, rows * max_ra) ||
            dalloc(&att, rows * max_att) || dalloc(&act, rows * max_ff) || dalloc(&proj, rows * max_proj) || dalloc(&qa, rows * max_q) ||
            dalloc(&gate, rows * max_heads) || dalloc(&z, rows * max_n) || dalloc(&rec, (size_t)gd_blocks((int)rows) * max_rec) ||
            dalloc(&fo, rows * max_n) || dalloc(&yf, rows * width) || dalloc(&part, (size_t)std::max(max_H, 1) * MAX_SPLIT * (max_dv + 2)) || dalloc(&inv, rows))
            return 1;
        cap = rows;
        return 0;
    }

    // every layer carries state that is not addressed by position: a step continues where the last one ended or starts a new
    // sequence at 0
    int begin_step(uint32_t pos, size_t n) override {
        if (pos != 0 && pos != next_pos) {
            error = "a model with recurrent layers continues at position " + std::to_string(next_pos) + " or restarts at 0, not at " + std::to_string(pos);
            return 1;
        }
        next_pos = pos + (uint32_t)n;
        return 0;
    }

    // ---- the residual stream ------------------------------------------------------------------------------------------------
    // what reads the residual stream next: a norm weight, and for a mixer the layer whose token shift follows the norm
    struct Next { const float* w = nullptr; const Layer* shift = nullptr; };
    Next mixer_of(size_t li) const { return li < layers.size() ? Next{layers[li].norm1, &layers[li]} : Next{}; }
    // x <- x + rms(yf) * wb (wb null: x as it is), then the next sublayer's input into h
    int residual_rows(cudaStream_t st, int T, const float* wb, const Next& nx, const PosSrc& ps) {
        ResNormRowsParams<AT> p{};
        p.y = yf; p.ldy = width; p.wb = wb; p.x = x; p.ldx = width; p.n = width; p.eps = info.eps; p.ps = ps;
        const bool two = nx.shift && T > 1;   // a row needs its neighbour's: factors first, then the shift
        if (two) p.inv_out = inv;
        else if (nx.w) {
            p.w_next = nx.w; p.h = h; p.ldh = width;
            if (nx.shift) { p.mu = nx.shift->mu; p.prev = nx.shift->prev; }
        }
        if (T == 1) {
            const int threads = std::min(1024, (width + 31) / 32 * 32);
            return launch_k("resnorm_rows_kernel", st, pdl_now, resnorm_rows_kernel<AT, true>, dim3(1), dim3(threads), 0, p);
        }
        if (launch_k("resnorm_rows_kernel", st, pdl_now, resnorm_rows_kernel<AT, false>, dim3(T), dim3(256), 0, p)) return 1;
        if (!two) return 0;
        NormShiftRowsParams<AT> sp{};
        sp.x = x; sp.ldx = width; sp.inv = inv; sp.w = nx.w; sp.mu = nx.shift->mu; sp.prev_in = nx.shift->prev; sp.prev_out = nx.shift->prev + layers.size() * width;
        sp.h = h; sp.ldh = width; sp.T = T; sp.n = width; sp.ps = ps;
        return launch_k("norm_shift_rows_kernel", st, pdl_now, norm_shift_rows_kernel<AT>, dim3((width + 255) / 256, (T + NORM_SHIFT_ROWS - 1) / NORM_SHIFT_ROWS),
                        dim3(256), 0, sp);
    }
    // a sublayer's last product a . w^T, its norm, the residual and the next sublayer's input
    int sublayer_out(cudaStream_t st, int T, const AT* a, int K, const WT* w, const float* wb, const Next& nx, const PosSrc& ps) {
        EpiParams<AT> e{}; e.out = yf; e.ldo = width; e.scale = 1.0f;
        if (this->template matmul<EPI_STORE>(st, T, a, K, w, nullptr, K, width, e)) return 1;
        return residual_rows(st, T, wb, nx, ps);
    }

    // ---- the layers -----------------------------------------------------------------------------------------------------------
    int in_proj(cudaStream_t st, const Layer& L, int T) {
        EpiParams<AT> e{}; e.out = proj; e.ldo = L.in_rows; e.scale = 1.0f;
        return this->template matmul<EPI_STORE>(st, T, h, width, L.w_in, nullptr, width, L.in_rows, e);
    }
    // the scan for a head size: rows per lane, lanes per column, columns and threads of a CTA follow from it
    static int scan_rows(int d) { return d <= 64 ? 64 : (d <= 128 ? 128 : (d <= 256 ? 256 : 512)); }
    template <int NR, int LPC, int CPT, int THREADS> int launch_scan(cudaStream_t st, const GeneralDeltaScanParams& sp) {
        constexpr int cols = THREADS / LPC * CPT;
        const size_t smem = general_delta_scan_smem<NR, LPC, CPT, THREADS>();
        if (optin(general_delta_scan_kernel<NR, LPC, CPT, THREADS>, smem)) return 1;
        return launch_k("general_delta_scan_kernel", st, pdl_now, general_delta_scan_kernel<NR, LPC, CPT, THREADS>, dim3((sp.d + cols - 1) / cols, sp.H), dim3(THREADS), smem, sp);
    }
    int scan(cudaStream_t st, const GeneralDeltaScanParams& sp) {
        switch (scan_rows(sp.d)) {
            case 64:
                if (scan_shape == 1) return launch_scan<2, 32, 2, 256>(st, sp);
                if (scan_shape == 2) return launch_scan<4, 16, 1, 256>(st, sp);
                return launch_scan<4, 16, 2, 128>(st, sp);
            case 128:
                if (scan_shape == 1) return launch_scan<4, 32, 2, 256>(st, sp);
                return launch_scan<8, 16, 2, 128>(st, sp);
            case 256: return launch_scan<8, 32, 2, 128>(st, sp);
            default: return launch_scan<16, 32, 1, 128>(st, sp);
        }
    }
    template <int RPT> int launch_step(cudaStream_t st, const GeneralDeltaStepParams<AT, WT>& p, int threads) {
        const size_t smem = ((size_t)p.ra + 5 * p.d + threads) * 4;
        if (optin(general_delta_step_kernel<AT, WT, RPT>, smem)) return 1;
        return launch_k("general_delta_step_kernel", st, pdl_now, general_delta_step_kernel<AT, WT, RPT>, dim3(p.H), dim3(threads), smem, p);
    }

    // leaves the row that the output projection multiplies in att
    int mixer_delta(cudaStream_t st, const Layer& L, int T, const PosSrc& ps) {
        const BoLayerCfg& c = L.c;
        const int n = c.H * c.d;
        if (in_proj(st, L, T)) return 1;
        if (T == 1 && step_fused) {
            GeneralDeltaStepParams<AT, WT> p{};
            p.proj = proj; p.w2 = L.w2; p.ra = c.ra; p.w0 = L.w0; p.a_bias = L.a_bias; p.w = L.onorm; p.eps = info.eps; p.state = L.state; p.out = att;
            p.H = c.H; p.d = c.d; p.decay_rate = decay_rate; p.ps = ps;
            p.cw = 32;
            while (p.cw < c.d) p.cw *= 2;
            const int threads = p.cw * std::min(1024 / p.cw, (c.d + 3) / 4);   // about four state rows per thread
            const int per = (c.d + threads / p.cw - 1) / (threads / p.cw);
            if (per <= 4) return launch_step<4>(st, p, threads);
            if (per <= 16) return launch_step<16>(st, p, threads);
            return launch_step<0>(st, p, threads);
        }
        CastColsParams<AT> cp{};   // the low-rank decay latent in the operand type, for the second half of that projection
        cp.in = proj + 5 * (size_t)n; cp.ld = L.in_rows; cp.out = lat; cp.ldo = c.ra; cp.n = c.ra; cp.total = T * c.ra; cp.tanh_first = 1;
        if (launch_k("cast_cols_kernel", st, pdl_now, cast_cols_kernel<AT>, dim3((cp.total + 255) / 256), dim3(256), 0, cp)) return 1;
        EpiParams<AT> ez{}; ez.out = z; ez.ldo = n; ez.scale = 1.0f; ez.bias = L.w0;
        if (this->template matmul<EPI_STORE>(st, T, lat, c.ra, L.w2, nullptr, c.ra, n, ez)) return 1;
        GeneralDeltaPreParams pp{};
        pp.proj = proj; pp.ld = L.in_rows; pp.z = z; pp.a_bias = L.a_bias; pp.rec = rec; pp.T = T; pp.H = c.H; pp.d = c.d; pp.dp = scan_rows(c.d); pp.decay_rate = decay_rate;
        if (launch_k("general_delta_pre_kernel", st, pdl_now, general_delta_pre_kernel, dim3(c.H, gd_blocks(T)), dim3(pp.dp), 0, pp)) return 1;
        GeneralDeltaScanParams sp{};
        sp.rec = rec; sp.state = L.state; sp.out = fo; sp.T = T; sp.H = c.H; sp.d = c.d; sp.ps = ps;
        if (scan(st, sp)) return 1;
        GatedHeadNormParams<AT> gp{};
        gp.o = fo; gp.graw = proj + 3 * (size_t)n; gp.w = L.onorm; gp.w_ld = c.d; gp.eps = info.eps; gp.out = att; gp.rows = T * c.H; gp.dv = c.d; gp.H = c.H;
        gp.g_ld = L.in_rows;
        return launch_k("gated_headnorm_kernel", st, pdl_now, gated_headnorm_kernel<AT>, dim3((gp.rows + 3) / 4), dim3(128), 0, gp);
    }

    int mixer_attention(cudaStream_t st, const Layer& L, int T, const PosSrc& ps, uint32_t pos_hint) {
        const BoLayerCfg& c = L.c;
        if (in_proj(st, L, T)) return 1;
        QkvPostParams qp{};
        qp.qkv = proj; qp.ld = L.in_rows; qp.H = c.H; qp.G = c.G; qp.dk = c.dk; qp.dv = c.dv; qp.q_only = c.kv_from >= 0;
        qp.qk_mode = c.rot_dims > 0 ? QK_ROTARY : QK_PLAIN; qp.eps = info.eps; qp.q_nw = L.qnorm; qp.k_nw = L.knorm;
        qp.rot_dims = c.rot_dims; qp.rot_cos = L.rot_cos; qp.rot_sin = L.rot_sin;
        qp.v_mode = V_PLAIN; qp.has_gate = true; qp.gate_out = gate; qp.q_out = qa; qp.kcache = L.kcache; qp.vcache = L.vcache; qp.ps = ps;
        const int tasks = c.H + 1 + (qp.q_only ? 0 : c.G + (c.G * c.dv + 127) / 128);
        const dim3 grid(T, T >= 64 ? std::min(4, (tasks + 3) / 4) : std::min(16, (tasks + 3) / 4));
        if (launch_k("qkv_post_kernel", st, pdl_now, qkv_post_kernel, grid, dim3(128), 0, qp)) return 1;
        AttnRowsParams<AT> p{};
        p.q = qa; p.kcache = L.kcache; p.vcache = L.vcache; p.out = att; p.gate = gate; p.wbias = L.wbias; p.chunk = c.chunk;
        p.T = T; p.H = c.H; p.G = c.G; p.dk = c.dk; p.dv = c.dv; p.scale = c.scale; p.ps = ps; p.k_ld = c.G * c.dk; p.v_ld = c.G * c.dv;
        return this->template attention_launch<true>(st, p, part, pos_hint);
    }

    int run_layers(cudaStream_t st, int T, const PosSrc& ps, uint32_t pos_hint) override {
        {
            EmbedRowsParams<WT> p{};
            p.embed = embed; p.bigram = nullptr; p.tokens = d_tokens; p.x = x; p.width = width; p.ps = ps;
            embed_rows_kernel<WT><<<T, 128, 0, st>>>(p);
            if (check_launch("embed_rows_kernel")) return 1;
        }
        if (residual_rows(st, T, nullptr, mixer_of(0), ps)) return 1;
        for (size_t li = 0; li < layers.size(); li++) {
            const Layer& L = layers[li];
            if (L.c.kind == BO_DELTA ? mixer_delta(st, L, T, ps) : mixer_attention(st, L, T, ps, pos_hint)) return 1;
            if (sublayer_out(st, T, att, L.wo_cols, L.wo, L.norm1b, L.c.ff > 0 ? Next{L.norm2, nullptr} : mixer_of(li + 1), ps)) return 1;
            if (L.c.ff > 0) {
                EpiParams<AT> eg{}; eg.act = act; eg.lda = L.c.ff; eg.glu_kind = GLU_SILU;
                if (this->template matmul<EPI_GLU>(st, T, h, width, L.wgate, L.wup, width, L.c.ff, eg)) return 1;
                if (sublayer_out(st, T, act, L.c.ff, L.wdown, L.norm2b, mixer_of(li + 1), ps)) return 1;
            }
            if (this->keep_layer(st, li, T)) return 1;
        }
        if (T > 1)   // the shift rows of all layers at once (one-row steps update them in place)
            GCK(cudaMemcpyAsync(shift_rows, shift_rows + layers.size() * width, layers.size() * width * 4, cudaMemcpyDeviceToDevice, st));
        return 0;
    }
    int head_rows(cudaStream_t st, int m, const uint32_t* rows_dev, float* out) override {
        EpiParams<AT> e{}; e.out = out; e.ldo = vocab; e.scale = 1.0f; e.softcap = softcap;
        if (m == 1 && rows_dev == nullptr) {
            GemvRowsParams<AT, WT> p{};
            p.x = x; p.nw = final_norm; p.eps = info.eps; p.w = head; p.K = width; p.O = vocab; p.e = e;
            return this->template launch_gemv<EPI_STORE, NORM_RMS>(st, p);
        }
        NormRowsParams<AT> np{};
        np.x = x; np.ldx = width; np.rows = rows_dev; np.w = final_norm; np.out = hn; np.ldo = width; np.n = width; np.eps = info.eps;
        if (launch_k("rmsnorm_rows_kernel", st, pdl_now, rmsnorm_rows_kernel<AT>, dim3(m), dim3(256), 0, np)) return 1;
        return this->template matmul<EPI_STORE>(st, m, hn, width, head, nullptr, width, vocab, e);
    }

    void set_model_option(const char* name, int value) override {
        if (!strcmp(name, "scan_shape")) { scan_shape = value; drop_graphs(); }
        if (!strcmp(name, "step_fused")) { step_fused = value; drop_graphs(); }
    }
    // test access: K and V rows of an attention layer (a borrower shows its lender's)
    int read_kv(cudaStream_t st, uint32_t layer, uint32_t pos0, uint32_t n, float* k_out, float* v_out) override {
        if (layer >= layers.size() || (size_t)pos0 + n > max_tokens) { error = "read_kv: out of range"; return 1; }
        const Layer& L = layers[layer];
        if (L.c.kind != BO_ATTENTION) { error = "read_kv: a delta-rule layer keeps a state, not rows per position"; return 1; }
        GCK(cudaStreamSynchronize(st));
        const size_t nk = (size_t)L.c.G * L.c.dk, nv = (size_t)L.c.G * L.c.dv;
        GCK(cudaMemcpy(k_out, L.kcache + pos0 * nk, n * nk * 4, cudaMemcpyDeviceToHost));
        GCK(cudaMemcpy(v_out, L.vcache + pos0 * nv, n * nv * 4, cudaMemcpyDeviceToHost));
        return 0;
    }
};

ArchModel* bolapel_factory(const std::string& dir, const Json& cfg, const ArchOptions& opt, std::string& err) {
    ArchModel* m = nullptr;
    int rc;
    if (opt.dtype == ARCH_F32) {
        auto* g = new BolapelModel<float, float>();
        rc = g->load(dir, cfg, opt);
        m = g;
    } else {
        auto* g = new BolapelModel<__nv_bfloat16, __nv_bfloat16>();
        rc = g->load(dir, cfg, opt);
        m = g;
    }
    if (rc) { err = m->error; delete m; return nullptr; }
    return m;
}

}  // namespace

void register_bolapel() { arch_register("Bolapel", bolapel_factory); }

}  // namespace lmrs
