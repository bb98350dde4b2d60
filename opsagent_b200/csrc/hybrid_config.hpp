// hybrid_config.hpp — configuration of the hybrid decoder family: a stack of parallel-residual layers whose token mixer is one of latent
// attention (a compressed key/value cache), a gated delta rule with per-channel decay, a Mamba-2 state-space layer, or windowed attention
// over cached keys and values (sliding window with optional kept first tokens, one or two score maps per head, optional sink, output gate,
// optionally reading another layer's cache), each beside a routed mixture-of-experts feed-forward, with an optional looped block that
// re-injects the embedding.  Six designs are registered: "Ratasun" (one weight-only layer norm per layer, sigmoid group-limited router, SwiGLU
// experts), "Zurevik" (two RMS norms per layer, softmax over the chosen router logits, squared-ReLU experts, scaled embedding, soft-capped
// logits) and "Rofizen" (norm after the sum: x <- norm(alpha x + sublayer(x)), mixer and feed-forward in sequence; mixers: gated linear
// attention with a decay per key channel, retention with a fixed decay per head and rotate-half rotary, or causal soft-capped attention with
// a distance penalty beside an xLSTM matrix memory; feed-forward: dense squared-ReLU, or SwiGLU experts chosen by a table of token ids plus
// a gated shared expert).  "Gosavik": pre-norm sublayers in sequence (x += mixer(rms1(x)), x += ff(rms2(x))) over several residual streams
// joined by learned coefficients (hyper-connections), a token shift in front of every mixer, a looped block without re-injection; mixers:
// latent attention with a low-rank query, rotate-half rotary with YaRN-scaled frequencies, a sliding window, a sink and a per-channel output
// gate, or causal grouped-query attention with projection biases, short convolutions on q / k / v, interleaved rotary, rotated values
// and a sink; feed-forward: dense with the tanh form of GELU.  "Petipel": sublayers in sequence with an RMS norm on either side of each
// (x += m norm(sublayer(norm(x))), factors stored as w - 1); mixers: causal grouped-query attention without rotation (a learned bias per
// head and distance bucket on the scores, a query temperature, values of unit RMS that later layers mix with the first layer's, a gate per
// head), or HGRN2 (a recurrence that writes with the complement of its forget gate); feed-forward: dense with PolyNorm, or experts with a
// clamped gated activation that are chosen by, and read their input times, a sigmoid score.  "Ketopel": plain pre-norm sublayers in sequence; mixers:
// latent attention with a sigmoid gate per head, a gated delta rule with one decay per head, or capped grouped-query attention (one norm over
// the whole query / key projection, rotate-half rotary with YaRN-scaled frequencies) beside lightning attention (a linear recurrence of activated
// queries, keys and values with a fixed decay per head, one norm over all heads), joined by two fixed factors; feed-forward: dense, gelu(gate) * up;
// a looped block that adds the embedding and a learned vector before its passes.
// Every size and constant is read from the checkpoint folder's config.json; nothing here is specific to one checkpoint.
#pragma once
#include <cstdio>
#include <fstream>
#include <sstream>
#include <stdexcept>
#include <string>
#include <vector>

#include "json_dom.hpp"

namespace oa {

enum HyMixer : int { HY_LATENT_ATTENTION = 0, HY_CHANNEL_DELTA = 1, HY_MAMBA2 = 2, HY_WINDOW_ATTENTION = 3, HY_LINEAR_ATTENTION = 4, HY_ATTENTION_BESIDE_MEMORY = 5 };
enum HyNorm : int { HY_LAYER_NORM = 0, HY_RMS_NORM = 1 };
enum HyRouterKind : int { HY_ROUTER_SIGMOID_GROUPS = 0, HY_ROUTER_SOFTMAX_CHOSEN = 1, HY_ROUTER_TOKEN_TABLE = 2, HY_ROUTER_SIGMOID_CHOSEN = 3 };   // weights: sigmoid scores renormalised and scaled / softmax over the chosen logits / a table row per token id, 1 / top each / the chosen logits' sigmoids as they are
// linear-attention recurrences over an fp32 state S[dim, vdim] per head, o_t = S_t^T q_t:
//   channel decay: S_t = diag(a_t) S_(t-1) + k_t v_t^T, a_t = sigmoid(z_t)^(1 / tau) per key channel from a low-rank projection (gated linear attention)
//   head decay:    S_t = decay_h S_(t-1) + k_t v_t^T with a fixed decay per head, rotate-half rotary on q and k (retention), or q = silu(.), k = silu(.), v = silu(.) (lightning attention)
//   forget write:  S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, f_t = l + (1 - l) sigmoid(z_t) per key channel with a lower bound l; q = silu(.), no keys (HGRN2)
//   matrix memory: S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k_t v_t^T with log gates i, f, a running maximum m and a normaliser n (xLSTM's mLSTM)
enum HyLinearKind : int { HY_LIN_CHANNEL_DECAY = 0, HY_LIN_HEAD_DECAY = 1, HY_LIN_MATRIX_MEMORY = 2, HY_LIN_FORGET_WRITE = 3 };
enum HyLinearNorm : int { HY_LIN_NORM_HEAD_WEIGHT = 0, HY_LIN_NORM_NONE = 1, HY_LIN_NORM_ALL_WEIGHT = 2, HY_LIN_NORM_JOINT = 3 };   // weight of the per-head RMS norm: [vdim] shared by heads / none / [heads * vdim]; or one RMS norm over all heads together, weight [heads * vdim]

struct HyLinear {
    int kind = HY_LIN_CHANNEL_DECAY, heads = 0, dim = 0, vdim = 0;
    float tau = 1.f, gate_cap = 0.f, rot_base = 10000.f; int rot_dims = 0;
    std::vector<float> decay;             // head decay: one per head
    int norm = HY_LIN_NORM_HEAD_WEIGHT, gate_silu = 1;      // output gate: silu (1) or sigmoid (0) of a projection, per channel (forget write: no output gate)
    bool q_scaled = true, k_scaled = false;                  // dim^-1/2 on q, or on k (after the rotation)
    bool qkv_silu = false;                                   // the projections of q, k and v pass a SiLU
};
// down(silu(gate x) * up x) / down(relu(up x)^2) / down(gelu_tanh(up x)) / down(g sigmoid(slope g) (u + 1)) with g = min(gate x, limit), u = clamp(up x, -limit, limit) /
// down(a N(z) + b N(z^2) + c N(z^3) + e) with z = up x and N(.) = unit RMS over the width (PolyNorm) / down(gelu_tanh(gate x) * up x)
enum HyExpertAct : int { HY_EXPERT_SWIGLU = 0, HY_EXPERT_RELU2 = 1, HY_EXPERT_GELU_TANH = 2, HY_EXPERT_CLAMPED_GLU = 3, HY_EXPERT_POLY_NORM = 4, HY_EXPERT_GELU_GLU = 5 };
constexpr float HY_CLAMPED_GLU_SLOPE = 1.702f;
enum HyRotLayout : int { HY_ROT_INTERLEAVED = 0, HY_ROT_HALVES = 1 };                         // channel 2i pairs with 2i + 1 / channel i with i + dims / 2
// YaRN: with where(t) = dims ln(original / (2 pi t)) / (2 ln base), lo = max(floor(where(fast)), 0), hi = min(ceil(where(slow)), dims - 1) and
// ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), frequency i is f_i / factor * ramp_i + f_i (1 - ramp_i); cos and sin carry the amplitude 0.1 ln(factor) + 1
struct HyRotScaling { bool on = false; float factor = 1.f, original = 0.f, fast = 0.f, slow = 0.f; };
enum HyGate : int { HY_GATE_NONE = 0, HY_GATE_CHANNEL = 1, HY_GATE_HEAD = 2 };

struct HyMoe {
    bool present = false;
    int experts = 0, top = 0, groups = 1, keep = 1, ff = 0;
    float scale = 1.f;
    int router = HY_ROUTER_SIGMOID_GROUPS, act = HY_EXPERT_SWIGLU;
    bool dense = false;                   // one feed-forward for every token (no router, no experts): down(act(up h)), width ff
    float limit = 0.f;                    // clamped gated activation
    bool weight_on_input = false;         // an expert reads weight * h, and its output is added as it is
    int shared_ff = 0;                    // > 0: a shared expert of this width runs for every token, times sigmoid(w_sg . h)
};

struct HyLayer {
    int type = HY_LATENT_ATTENTION;
    // latent attention: heads x (dim unrotated + rot_dim rotated) query/key, vdim values, kv_rank latent; rotary on the first rot_dims of the rotated part
    // channel delta:    heads value heads of vdim, kv_heads query/key heads of dim, conv taps; head_decay: one decay per head and a full-rank SiLU gate
    //                   instead of a decay per key channel and a low-rank sigmoid gate
    // mamba2:           heads x vdim inner channels, state N, groups of B/C, norm_groups, conv taps
    int heads = 0, kv_heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, rot_dims = 0, conv = 0, state = 0, groups = 1, norm_groups = 1;
    float rot_base = 10000.f, scale = 1.f;
    // window attention: heads query heads on kv_heads key/value heads, `maps` score maps per head (2 = differential: q and k hold [map 1 | map 2] per
    // head, out = a1 - lambda a2, unit RMS per head, times 1 - diff); position i sees j <= i with i - j < window or j < keep_first; qk_norm: RMS
    // norm of every query / key map with a weight shared by heads and maps; bias: q/k/v projection biases; sink: a learned logit per head in
    // the softmax denominator only; gate: sigmoid output gate per channel or per head; kv_from >= 0: keys and values of that layer's cache
    // qk_norm = 2: one RMS norm over the whole q (and k) projection, before the split into heads, with a weight of that size.  softcap > 0:
    // score <- softcap tanh(score / softcap).  slope_exp > 0: head h's score loses 2^(-slope_exp (h + 1) / heads) per position of distance.
    // q_temp_every > 0: q at position p is multiplied by 1 + q_temp_coef ln(floor((p + 1) / q_temp_every) + 1).  out_bias: bias of the output projection
    int maps = 1, window = 0, keep_first = 0, qk_norm = 0, bias = 0, sink = 0, gate = HY_GATE_NONE, kv_from = -1;
    float diff = 0.f, softcap = 0.f, slope_exp = 0.f, q_temp_coef = 0.f; int q_temp_every = 0, out_bias = 0;
    // latent attention, optional parts: q_rank > 0: queries through a latent, q = W_uq rms_norm(W_dq h); rot_layout / rot_scaling: pairing and
    // YaRN scaling of the rotary; window > 0: position i sees j with 0 <= i - j < window; sink; gate: sigmoid(W_g h) per channel or per head.
    // windowed attention, optional parts: conv > 0: a short causal convolution (no bias, no activation) on every channel of q, k and v, right
    // after the projection; rot_dims > 0: rotary on the first rot_dims channels of every query / key head; v_rot: the value of position j is
    // cached turned by j over all vdim channels (pair m by j rot_base^(-2m / vdim)), a head's output at position i is turned back by -i
    // bias_max > 0: a learned bias per head and distance bucket is added to the scaled score: with B table rows, distances below B / 2 have a row
    // each, then a logarithmic scale up to bias_max, the last row beyond.  v_norm: a value head is cached divided by its RMS.  v_mix: every
    // such layer but the first caches (1 - lambda) v + lambda v_first, v_first = the first such layer's cached value of the same token (v_first: its layer, -1: this is the first)
    int bias_max = 0, v_norm = 0, v_mix = 0, v_first = -1;
    int q_rank = 0, rot_layout = HY_ROT_INTERLEAVED, v_rot = 0, head_decay = 0;
    // attention beside a linear recurrence (HY_ATTENTION_BESIDE_MEMORY): scaled_sum: the two outputs are joined as left_scale * left + right_scale * right
    // instead of the halves of their RMS norms; rot_dims > 0: rotary on the attention side's queries and keys, after their norm
    bool scaled_sum = false; float left_scale = 1.f, right_scale = 1.f;
    HyRotScaling rot_scaling;
    HyLinear lin;                         // HY_LINEAR_ATTENTION, and the memory side of HY_ATTENTION_BESIDE_MEMORY (whose attention side uses the fields above)
    HyMoe moe;
};

struct HyRun { int layer = 0, pass = -1; bool first_of_pass = false; int cache_idx = -1, state_idx = -1; bool cache_owner = false; int index = 0; };   // one execution of a layer (a looped layer runs once per pass)

struct HybridConfig {
    std::string dir;                      // checkpoint folder (config.json [+ model.safetensors]; without the latter the weights are seeded)
    int width = 0, vocab = 0;
    float eps = 1e-6f, logit_scale = 1.f;
    std::string arch = "ratasun";        // registry key of the design
    int norm = HY_LAYER_NORM;             // the layers' (and the final) norm
    bool two_norms = false;               // mixer and feed-forward each read their own norm of the same residual
    float embed_scale = 1.f, logit_softcap = 0.f;      // x = embed[token] * scale; logits <- cap * tanh(logits / cap) (0: none)
    bool post_norm = false; float post_alpha = 1.f;    // norm after the sum: x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)); the sublayers read x itself
    // sublayers in sequence, each on its own norm of the residual it finds: x <- x + mixer(norm1(x)), then x <- x + ff(norm2(x)).
    // streams > 0 (hyper-connections): the residual is `streams` copies x_1..x_s of the embedding; sublayer q reads u = sum_s in_q[s] x_s and
    // every stream becomes x_t <- sum_s mix_q[s, t] x_s + out_q[t] sublayer(norm(u)); after the last layer x = sum_s x_s.
    // token_shift: the mixer's input h_t (after the norm) is replaced by h_t + (h_(t-1) - h_t) * shift, h_(t-1) as it was before its own
    // replacement (zeros before the first token); every layer execution carries the last h of a sequence in its state slot.
    bool sequential = false, token_shift = false; int streams = 0;
    // branch_norm (sequential designs): a sublayer's output passes a norm of its own before it joins the residual: x <- x + residual_mult norm_b(sublayer(norm(x))).
    // norm_around_zero: the layers' and the final norm weights are stored as w - 1
    bool branch_norm = false, norm_around_zero = false; float residual_mult = 1.f;
    bool loop_reinject = true;                          // a looped block re-injects the embedding before every pass (x <- W_in [x ; x0] + step[pass])
    bool loop_add = false;                              // ... or adds it: before every pass but the first x <- x + x0, before every pass x <- x + step[pass]
    bool single_stream = false;                         // sequential designs: one residual, sublayers' outputs join it as they are
    std::vector<HyLayer> layers;
    int loop_start = 0, loop_stop = 0, loop_times = 0;    // times == 0: no looped block
    std::vector<HyRun> runs;
    int n_caches = 0, n_states = 0;

    static double num(const Json& o, const char* k, const char* where) {
        const Json* j = o.get(k);
        if (!j || j->t != Json::Num) throw std::runtime_error(std::string("config.json: ") + where + " needs a number '" + k + "'");
        return j->n;
    }
    static int integer(const Json& o, const char* k, const char* where) { return (int)std::llround(num(o, k, where)); }
    static const Json& obj(const Json& o, const char* k, const char* where) {
        const Json* j = o.get(k);
        if (!j || j->t != Json::Obj) throw std::runtime_error(std::string("config.json: ") + where + " needs an object '" + k + "'");
        return *j;
    }

    static std::string read_file(const std::string& path) {
        std::ifstream f(path, std::ios::binary);
        if (!f) throw std::runtime_error("cannot read " + path);
        std::stringstream ss; ss << f.rdbuf(); return ss.str();
    }
    // the "architecture" key of <dir>/config.json (empty if there is none): the model registry dispatches on it
    static std::string architecture_of(const std::string& dir) {
        Json j; std::string err;
        if (!parse_json(read_file(dir + "/config.json"), j, err)) throw std::runtime_error("config.json: " + err);
        return j.str("architecture");
    }

    // the model registry of this family: config.json's "architecture" -> registry key ("" = not one of ours)
    static std::string registry_key(const std::string& architecture) {
        if (architecture == "Ratasun") return "ratasun";
        if (architecture == "Zurevik") return "zurevik";
        if (architecture == "Rofizen") return "rofizen";
        if (architecture == "Gosavik") return "gosavik";
        if (architecture == "Petipel") return "petipel";
        if (architecture == "Ketopel") return "ketopel";
        return "";
    }

    static HybridConfig load(const std::string& dir) {
        Json j; std::string err;
        if (!parse_json(read_file(dir + "/config.json"), j, err)) throw std::runtime_error("config.json: " + err);
        HybridConfig c; c.dir = dir;
        c.arch = registry_key(j.str("architecture"));
        if (c.arch.empty()) throw std::runtime_error("config.json: unknown architecture '" + j.str("architecture") + "'");
        const bool zu = c.arch == "zurevik", ro = c.arch == "rofizen", go = c.arch == "gosavik", pe = c.arch == "petipel", ke = c.arch == "ketopel";
        if (ke) { c.norm = HY_RMS_NORM; c.sequential = true; c.single_stream = true; c.loop_reinject = false; c.loop_add = true; }
        if (go) {
            c.norm = HY_RMS_NORM; c.sequential = true; c.token_shift = true; c.loop_reinject = false;
            if (j.get("streams") && j.get("streams")->t == Json::Num) { c.streams = integer(j, "streams", "the model"); if (c.streams < 1 || c.streams > 8) throw std::runtime_error("config.json: streams must be 1 .. 8"); }
        }
        if (pe) {
            c.norm = HY_RMS_NORM; c.sequential = true; c.branch_norm = true; c.norm_around_zero = true; c.loop_reinject = false;
            c.residual_mult = (float)num(j, "residual_mult", "the model");
        }
        if (zu) { c.norm = HY_RMS_NORM; c.two_norms = true; }
        if (ro) { c.post_norm = true; c.post_alpha = (float)num(j, "postln_alpha", "the model"); }
        if (const Json* e = j.get("embedding")) if (e->t == Json::Obj && e->get("scale")) c.embed_scale = (float)num(*e, "scale", "embedding");
        if (j.get("logit_softcap") && j.get("logit_softcap")->t == Json::Num) c.logit_softcap = (float)num(j, "logit_softcap", "the model");
        c.width = integer(j, "width", "the model"); c.vocab = integer(j, "vocab", "the model");
        c.eps = (float)num(obj(j, "norm", "the model"), "eps", "norm");
        c.logit_scale = j.get("logit_scale") ? (float)num(j, "logit_scale", "the model") : 1.f;
        const Json* ls = j.get("layers");
        if (!ls || ls->t != Json::Arr || ls->a.empty()) throw std::runtime_error("config.json: 'layers' must be a non-empty list");
        auto read_scaling = [](HyLayer& l, const Json& rot) {        // optional YaRN scaling of a rotary
            const Json* sc = rot.get("scaling");
            if (!sc || sc->t != Json::Obj) return;
            l.rot_scaling.on = true; l.rot_scaling.factor = (float)num(*sc, "factor", "scaling"); l.rot_scaling.original = (float)num(*sc, "original", "scaling");
            l.rot_scaling.fast = (float)num(*sc, "fast", "scaling"); l.rot_scaling.slow = (float)num(*sc, "slow", "scaling");
            if (!(l.rot_scaling.factor > 0.f) || !(l.rot_scaling.original > 0.f) || !(l.rot_scaling.fast > 0.f) || !(l.rot_scaling.slow > 0.f) || !(l.rot_base > 1.f))
                throw std::runtime_error("config.json: bad rotary scaling");
        };
        auto read_decay = [](HyLinear& n, const Json& m, const char* where) {        // a fixed decay per head
            const Json* d = m.get("decay");
            if (!d || d->t != Json::Arr || (int)d->a.size() != n.heads) throw std::runtime_error(std::string("config.json: ") + where + " needs a list 'decay' with one number per head");
            for (const Json& x : d->a) { if (x.t != Json::Num) throw std::runtime_error("config.json: 'decay' holds numbers"); n.decay.push_back((float)x.n); }
        };
        for (const Json& lj : ls->a) {
            HyLayer l; const std::string type = lj.str("type");
            const Json& m = obj(lj, "mixer", "a layer");
            if (type == "latent_attention") {
                l.type = HY_LATENT_ATTENTION;
                l.heads = integer(m, "heads", type.c_str()); l.dim = integer(m, "dim", type.c_str()); l.rot_dim = integer(m, "rot_dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.kv_rank = integer(m, "kv_rank", type.c_str()); l.scale = (float)num(m, "scale", type.c_str());
                const Json& r = obj(m, "rot", type.c_str());
                l.rot_base = (float)num(r, "base", "rot"); l.rot_dims = integer(r, "dims", "rot");
                if (l.rot_dims > l.rot_dim || (l.rot_dims & 1)) throw std::runtime_error("config.json: rot.dims must be even and <= rot_dim");
                if (go) {
                    l.q_rank = integer(m, "q_rank", type.c_str()); l.rot_layout = HY_ROT_HALVES; l.sink = 1; l.gate = HY_GATE_CHANNEL;
                    if (const Json* mk = m.get("mask")) if (mk->t == Json::Obj) { l.window = integer(*mk, "size", "mask"); if (l.window < 1) throw std::runtime_error("config.json: mask.size must be at least 1"); }
                    read_scaling(l, r);
                    if (l.q_rank <= 0 || l.dim < 0 || l.rot_dim < 0 || l.dim + l.rot_dim <= 0 || l.kv_rank <= 0 || l.kv_rank > 1024) throw std::runtime_error("config.json: bad latent attention sizes");
                }
                if (ke) {
                    l.gate = HY_GATE_HEAD; read_scaling(l, r);
                    if (l.dim < 0 || l.rot_dim < 0 || l.dim + l.rot_dim <= 0 || l.rot_dims < 0 || l.kv_rank <= 0 || l.kv_rank > 1024 || !(l.rot_base > 0.f)) throw std::runtime_error("config.json: bad latent attention sizes");
                }
            } else if (!ke && type == "channel_delta") {
                l.type = HY_CHANNEL_DELTA;
                l.heads = integer(m, "heads", type.c_str()); l.kv_heads = integer(m, "kv_heads", type.c_str()); l.dim = integer(m, "dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.conv = integer(m, "conv", type.c_str());
                if (l.kv_heads <= 0 || l.heads % l.kv_heads) throw std::runtime_error("config.json: kv_heads must divide heads");
            } else if (ke && type == "delta") {
                l.type = HY_CHANNEL_DELTA; l.head_decay = 1;
                l.heads = integer(m, "heads", type.c_str()); l.kv_heads = integer(m, "kv_heads", type.c_str()); l.dim = integer(m, "dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.conv = integer(m, "conv", type.c_str());
                if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.dim > 760) throw std::runtime_error("config.json: bad delta-rule sizes");
            } else if (ke && type == "parallel") {
                // causal capped attention (left) beside lightning attention (right), both reading the layer's normed input
                l.type = HY_ATTENTION_BESIDE_MEMORY; l.scaled_sum = true;
                const Json& a = obj(m, "left", "parallel"); const Json& b = obj(m, "right", "parallel");
                l.heads = integer(a, "heads", "left"); l.kv_heads = integer(a, "kv_heads", "left"); l.dim = integer(a, "dim", "left"); l.vdim = integer(a, "vdim", "left");
                l.scale = (float)num(a, "scale", "left"); l.window = 1 << 30; l.qk_norm = 2;
                l.left_scale = (float)num(m, "left_scale", "parallel"); l.right_scale = (float)num(m, "right_scale", "parallel");
                if (a.get("softcap") && a.get("softcap")->t == Json::Num) l.softcap = (float)num(a, "softcap", "left");          // absent or 0: scores are not capped
                const Json& r = obj(a, "rot", "left");
                l.rot_base = (float)num(r, "base", "rot"); l.rot_dims = integer(r, "dims", "rot"); l.rot_layout = HY_ROT_HALVES; read_scaling(l, r);
                if (l.heads <= 0 || l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.vdim > 256 || l.dim > 1024 || l.softcap < 0.f || l.rot_dims < 0 || l.rot_dims > l.dim || (l.rot_dims & 1) || !(l.rot_base > 0.f))
                    throw std::runtime_error("config.json: bad attention sizes");
                HyLinear& n = l.lin;
                n.kind = HY_LIN_HEAD_DECAY; n.heads = integer(b, "heads", "right"); n.dim = integer(b, "dim", "right"); n.vdim = integer(b, "vdim", "right");
                n.norm = HY_LIN_NORM_JOINT; n.gate_silu = 0; n.q_scaled = false; n.qkv_silu = true;
                read_decay(n, b, "lightning attention");
                if (n.heads <= 0 || n.dim <= 0 || n.dim > 760 || n.vdim <= 0) throw std::runtime_error("config.json: bad linear-attention sizes");
            } else if (!ke && type == "mamba2") {
                l.type = HY_MAMBA2;
                l.heads = integer(m, "heads", type.c_str()); l.vdim = integer(m, "vdim", type.c_str()); l.state = integer(m, "state", type.c_str());
                l.groups = integer(m, "groups", type.c_str()); l.norm_groups = integer(m, "norm_groups", type.c_str()); l.conv = integer(m, "conv", type.c_str());
                if (l.groups <= 0 || l.heads % l.groups || l.norm_groups <= 0 || (l.heads * l.vdim) % l.norm_groups) throw std::runtime_error("config.json: groups must divide heads, norm_groups the inner size");
            } else if (go && type == "attention") {
                // causal grouped-query attention: projection biases, short convolutions, interleaved rotary on queries and keys, rotated values, a sink per head
                l.type = HY_WINDOW_ATTENTION;
                l.heads = integer(m, "heads", type.c_str()); l.kv_heads = integer(m, "kv_heads", type.c_str()); l.dim = integer(m, "dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.scale = (float)num(m, "scale", type.c_str()); l.conv = integer(m, "conv", type.c_str());
                const Json& r = obj(m, "rot", type.c_str());
                l.rot_base = (float)num(r, "base", "rot"); l.rot_dims = integer(r, "dims", "rot"); l.rot_layout = HY_ROT_INTERLEAVED;
                l.window = 1 << 30; l.bias = 1; l.out_bias = 1; l.sink = 1; l.v_rot = 1;
                if (const Json* mk = m.get("mask")) if (mk->t == Json::Obj) { l.window = integer(*mk, "size", "mask"); if (l.window < 1) throw std::runtime_error("config.json: mask.size must be at least 1"); }
                if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.vdim > 256 || (l.vdim & 1) || l.dim > 1024 || l.rot_dims < 0 || l.rot_dims > l.dim || (l.rot_dims & 1) || l.conv < 1 || l.conv > 16 || !(l.rot_base > 0.f))
                    throw std::runtime_error("config.json: bad attention sizes");
            } else if (pe && type == "attention") {
                // causal grouped-query attention, no rotation: distance bias, query temperature, unit-RMS values mixed with the first such layer's, a gate per head
                l.type = HY_WINDOW_ATTENTION;
                l.heads = integer(m, "heads", type.c_str()); l.kv_heads = integer(m, "kv_heads", type.c_str()); l.dim = integer(m, "dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.scale = (float)num(m, "scale", type.c_str()); l.bias_max = integer(m, "bias_max", type.c_str());
                l.window = 1 << 30; l.gate = HY_GATE_HEAD; l.v_norm = 1;
                if (const Json* qt = m.get("q_temp")) if (qt->t == Json::Obj) { l.q_temp_coef = (float)num(*qt, "coef", "q_temp"); l.q_temp_every = integer(*qt, "every", "q_temp"); if (l.q_temp_every < 1) throw std::runtime_error("config.json: q_temp.every must be at least 1"); }
                if (const Json* vm = m.get("v_mix")) l.v_mix = (vm->t == Json::Bool && vm->b) || (vm->t == Json::Num && vm->n != 0);
                if (l.v_mix) for (int i = 0; i < (int)c.layers.size() && l.v_first < 0; ++i) if (c.layers[i].v_mix) {
                    l.v_first = i;
                    if (c.layers[i].kv_heads != l.kv_heads || c.layers[i].vdim != l.vdim) throw std::runtime_error("config.json: layers that mix values need the same kv_heads and vdim");
                }
                if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.vdim > 256 || l.dim > 1024 || l.bias_max < 1 || l.bias_max > (1 << 22)) throw std::runtime_error("config.json: bad attention sizes");
            } else if (pe && type == "hgrn2") {
                l.type = HY_LINEAR_ATTENTION; HyLinear& n = l.lin;
                n.heads = l.heads = integer(m, "heads", type.c_str()); n.dim = l.dim = integer(m, "dim", type.c_str()); n.vdim = l.vdim = integer(m, "vdim", type.c_str());
                n.kind = HY_LIN_FORGET_WRITE; n.norm = HY_LIN_NORM_HEAD_WEIGHT; n.q_scaled = false;
                if (n.dim <= 0 || n.dim > 768) throw std::runtime_error("config.json: bad linear-attention sizes");
            } else if (!pe && !ke && (type == "attention" || type == "attention_2")) {
                // "attention": differential (two score maps), query/key norm, kept first tokens, gate per channel;
                // "attention_2": one map, projection biases, a sink per head, gate per head, optionally another layer's keys and values
                const bool diff = type == "attention";
                l.type = HY_WINDOW_ATTENTION;
                l.heads = integer(m, "heads", type.c_str()); l.kv_heads = integer(m, "kv_heads", type.c_str()); l.dim = integer(m, "dim", type.c_str());
                l.vdim = integer(m, "vdim", type.c_str()); l.scale = (float)num(m, "scale", type.c_str());
                const Json& mk = obj(m, "mask", type.c_str());
                l.window = integer(mk, "size", "mask");
                if (mk.get("keep_first") && mk.get("keep_first")->t == Json::Num) l.keep_first = integer(mk, "keep_first", "mask");
                l.maps = diff ? 2 : 1; l.qk_norm = diff; l.bias = !diff; l.sink = !diff; l.gate = diff ? HY_GATE_CHANNEL : HY_GATE_HEAD;
                if (diff) l.diff = (float)num(m, "diff", type.c_str());
                if (!diff && m.get("kv_from") && m.get("kv_from")->t == Json::Num) {
                    l.kv_from = integer(m, "kv_from", type.c_str());
                    if (l.kv_from < 0 || l.kv_from >= (int)c.layers.size()) throw std::runtime_error("config.json: kv_from must name an earlier layer");
                    const HyLayer& src = c.layers[l.kv_from];
                    if (src.type != HY_WINDOW_ATTENTION || src.kv_from >= 0 || src.maps != l.maps || src.kv_heads != l.kv_heads || src.dim != l.dim || src.vdim != l.vdim)
                        throw std::runtime_error("config.json: kv_from must name a layer with keys and values of its own and of this layer's sizes");
                }
                if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.window < 1 || l.keep_first < 0 || l.vdim > 256 || l.dim > 1024) throw std::runtime_error("config.json: bad attention sizes");
            } else if (ro && (type == "gla" || type == "retention")) {
                l.type = HY_LINEAR_ATTENTION; HyLinear& n = l.lin;
                n.heads = l.heads = integer(m, "heads", type.c_str()); n.dim = l.dim = integer(m, "dim", type.c_str()); n.vdim = l.vdim = integer(m, "vdim", type.c_str());
                if (type == "gla") { n.kind = HY_LIN_CHANNEL_DECAY; n.tau = (float)num(m, "tau", "gla"); n.norm = HY_LIN_NORM_HEAD_WEIGHT; if (!(n.tau > 0.f)) throw std::runtime_error("config.json: gla needs tau > 0"); }
                else {
                    n.kind = HY_LIN_HEAD_DECAY; n.norm = HY_LIN_NORM_NONE; n.q_scaled = false; n.k_scaled = true;
                    read_decay(n, m, "retention");
                    const Json& r = obj(m, "rot", "retention");
                    n.rot_base = (float)num(r, "base", "rot"); n.rot_dims = integer(r, "dims", "rot");
                    if (n.rot_dims < 0 || n.rot_dims > n.dim || (n.rot_dims & 1)) throw std::runtime_error("config.json: rot.dims must be even and <= dim");
                }
                if (n.dim <= 0 || n.dim > 1024) throw std::runtime_error("config.json: bad linear-attention sizes");
            } else if (ro && type == "parallel") {
                // causal attention (left) beside a matrix memory (right), both reading the layer's input; the halves of their RMS-normed outputs are added
                l.type = HY_ATTENTION_BESIDE_MEMORY;
                const Json& a = obj(m, "left", "parallel"); const Json& b = obj(m, "right", "parallel");
                l.heads = integer(a, "heads", "left"); l.kv_heads = integer(a, "kv_heads", "left"); l.dim = integer(a, "dim", "left"); l.vdim = integer(a, "vdim", "left");
                l.scale = (float)num(a, "scale", "left"); l.slope_exp = 8.f;
                if (a.get("softcap") && a.get("softcap")->t == Json::Num) l.softcap = (float)num(a, "softcap", "left");          // absent or 0: scores are not capped
                if (const Json* qt = a.get("q_temp")) if (qt->t == Json::Obj) { l.q_temp_coef = (float)num(*qt, "coef", "q_temp"); l.q_temp_every = integer(*qt, "every", "q_temp"); if (l.q_temp_every < 1) throw std::runtime_error("config.json: q_temp.every must be at least 1"); }
                l.window = 1 << 30; l.qk_norm = 2; l.bias = 1; l.out_bias = 1;
                if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.dim <= 0 || l.vdim > 256 || l.dim > 1024 || l.softcap < 0.f) throw std::runtime_error("config.json: bad attention sizes");
                HyLinear& n = l.lin;
                n.kind = HY_LIN_MATRIX_MEMORY; n.heads = integer(b, "heads", "right"); n.dim = integer(b, "dim", "right"); n.vdim = integer(b, "vdim", "right");
                n.gate_cap = (float)num(b, "gate_cap", "right"); n.norm = HY_LIN_NORM_ALL_WEIGHT; n.gate_silu = 0;
                if (n.heads <= 0 || n.dim <= 0 || n.dim > 1024 || n.vdim <= 0 || !(n.gate_cap > 0.f)) throw std::runtime_error("config.json: bad matrix-memory sizes");
            } else throw std::runtime_error("config.json: unknown layer type '" + type + "'");
            const bool recurrent = l.type == HY_CHANNEL_DELTA || l.type == HY_MAMBA2;
            if (l.heads <= 0 || l.vdim <= 0 || (recurrent && (l.conv < 1 || l.conv > 16))) throw std::runtime_error("config.json: bad mixer sizes");
            const Json* mj = lj.get("mlp");
            if (mj && mj->t == Json::Obj && (ro || go || pe || ke) && mj->str("kind") == "dense") {
                l.moe.present = true; l.moe.dense = true; l.moe.act = ke ? HY_EXPERT_GELU_GLU : pe ? HY_EXPERT_POLY_NORM : go ? HY_EXPERT_GELU_TANH : HY_EXPERT_RELU2; l.moe.experts = 1; l.moe.top = 1;
                l.moe.ff = integer(*mj, "ff", "mlp");
                if (l.moe.ff <= 0) throw std::runtime_error("config.json: bad feed-forward width");
            } else if (mj && mj->t == Json::Obj) {
                if (go || ke || mj->str("kind") != "moe") throw std::runtime_error("config.json: unknown mlp kind '" + mj->str("kind") + "'");
                const Json& r = obj(*mj, "router", "mlp");
                l.moe.present = true; l.moe.ff = integer(obj(*mj, "expert", "mlp"), "ff", "expert");
                l.moe.experts = integer(r, "experts", "router"); l.moe.top = integer(r, "top", "router");
                if (pe) {
                    l.moe.router = HY_ROUTER_SIGMOID_CHOSEN; l.moe.act = HY_EXPERT_CLAMPED_GLU; l.moe.weight_on_input = true; l.moe.limit = (float)num(obj(*mj, "expert", "mlp"), "limit", "expert");
                    if (l.moe.ff <= 0 || !(l.moe.limit > 0.f)) throw std::runtime_error("config.json: bad expert sizes");
                }
                else if (zu) { l.moe.router = HY_ROUTER_SOFTMAX_CHOSEN; l.moe.act = HY_EXPERT_RELU2; }
                else if (ro) {
                    l.moe.router = HY_ROUTER_TOKEN_TABLE;
                    if (const Json* sh = mj->get("shared")) if (sh->t == Json::Obj) { l.moe.shared_ff = integer(*sh, "ff", "shared"); if (l.moe.shared_ff <= 0) throw std::runtime_error("config.json: bad shared expert width"); }
                    if (l.moe.ff <= 0) throw std::runtime_error("config.json: bad expert width");
                }
                else l.moe.scale = (float)num(r, "scale", "router");
                if (const Json* g = r.get("groups")) if (g->t == Json::Obj) { l.moe.groups = integer(*g, "count", "groups"); l.moe.keep = integer(*g, "keep", "groups"); }
                if (l.moe.groups <= 0 || l.moe.experts % l.moe.groups || l.moe.keep <= 0 || l.moe.keep > l.moe.groups || l.moe.top <= 0 ||
                    l.moe.top > l.moe.keep * (l.moe.experts / l.moe.groups) || l.moe.top > 31 + (l.moe.shared_ff ? 0 : 1) || l.moe.experts > 1024)
                    throw std::runtime_error("config.json: bad router sizes");
            }
            c.layers.push_back(l);
        }
        const Json* lp = j.get("loop");
        if (lp && lp->t == Json::Obj) {
            c.loop_start = integer(*lp, "start", "loop"); c.loop_stop = integer(*lp, "stop", "loop"); c.loop_times = integer(*lp, "times", "loop");
            if (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > (int)c.layers.size() || c.loop_times < 1) throw std::runtime_error("config.json: bad loop");
        }
        // expand the schedule of layer executions: each execution owns its cache (attention) or state (recurrent mixers)
        auto add = [&](int layer, int pass, bool first) {
            HyRun r; r.layer = layer; r.pass = pass; r.first_of_pass = first;
            const HyLayer& l = c.layers[layer];
            if (l.type == HY_WINDOW_ATTENTION && l.kv_from >= 0) {          // the cache of the (only) execution of the layer it reads
                for (const HyRun& o : c.runs) if (o.layer == l.kv_from) r.cache_idx = o.cache_idx;
                if (r.cache_idx < 0 || (c.loop_times > 0 && layer >= c.loop_start && layer < c.loop_stop) || (c.loop_times > 0 && l.kv_from >= c.loop_start && l.kv_from < c.loop_stop))
                    throw std::runtime_error("config.json: a layer that reads another layer's cache cannot be part of a looped block");
            } else if (l.type == HY_LATENT_ATTENTION || l.type == HY_WINDOW_ATTENTION) {
                r.cache_idx = c.n_caches++; r.cache_owner = true;
                if (l.type == HY_WINDOW_ATTENTION && l.conv > 1) r.state_idx = c.n_states++;        // the convolutions' tails
            }
            else if (l.type == HY_ATTENTION_BESIDE_MEMORY) { r.cache_idx = c.n_caches++; r.cache_owner = true; r.state_idx = c.n_states++; }     // a cache for the attention side, a state for the memory side
            else r.state_idx = c.n_states++;
            r.index = (int)c.runs.size();
            c.runs.push_back(r);
        };
        for (int i = 0; i < (int)c.layers.size();) {
            if (c.loop_times > 0 && i == c.loop_start) {
                for (int t = 0; t < c.loop_times; ++t) for (int k = c.loop_start; k < c.loop_stop; ++k) add(k, t, k == c.loop_start);
                i = c.loop_stop;
            } else { add(i, -1, false); ++i; }
        }
        if (c.width <= 0 || c.vocab <= 0) throw std::runtime_error("config.json: bad width / vocab");
        return c;
    }
};

}  // namespace oa
