// HuggingFace config.json -> model IR. One IR layer per logical op, parameters named exactly as in
// the HF safetensors files so that the weight sharder can slice checkpoints by name:
//   0            Embedding
//   4i+1..4i+4   RmsNorm(input_layernorm), Attention(self_attn), RmsNorm(post_attention_layernorm),
//                Moe(block_sparse_moe) or Mlp(mlp)                    for block i
//   4N+1, 4N+2   RmsNorm(model.norm), Lmhead
// The reference builds the same list for Mixtral (crates/skein_ir/src/model/mixtral.rs:74-372) and
// rejects every other architecture (model/mod.rs:33-47); the Llama family (Llama, Mistral, Qwen2
// shapes) is imported here as well.
#pragma once
#include "ir.hpp"

namespace skein {

inline size_t cfg_usize(const Json& j, const char* k) {
  const Json* v = j.find(k);
  if (!v || v->is_null()) throw ImportError(std::string("config.json: missing `") + k + "`");
  long long x = v->as_int();
  if (x < 0) throw ImportError(std::string("config.json: `") + k + "` is negative");
  return (size_t)x;
}

// A design that lists its layers one by one (Zarorax): post-norm blocks of latent attention and a dense or routed
// feed-forward, each with sizes of its own. The tensor names are those of the checkpoint ("l<i>.mix.dkv", "l<i>.mlp.e0.up").
// A block with `weights_of` has no parameters; what it streams is counted in shared_elems.
inline Graph import_layered(const Json& cfg) {
  ModelMeta m;
  m.architecture = cfg.at("architecture").as_string();
  m.layered = true;
  m.hidden = cfg_usize(cfg, "width");
  m.vocab = cfg_usize(cfg, "vocab");
  m.max_position = cfg.has("max_position_embeddings") && !cfg.at("max_position_embeddings").is_null() ? cfg_usize(cfg, "max_position_embeddings") : 131072;
  for (const char* k : {"norm", "canon", "postln_alpha", "layers"})
    if (!cfg.has(k)) throw ImportError(std::string("config.json: missing `") + k + "`");
  m.rms_norm_eps = cfg.at("norm").at("eps").as_double();
  const size_t taps = cfg_usize(cfg.at("canon"), "taps");
  const auto& layers = cfg.at("layers").items();
  if (layers.empty()) throw ImportError("config.json: `layers` is empty");
  m.num_layers = layers.size();
  m.num_kv_heads = 1;
  Graph g;
  size_t idx = 0;
  const uint64_t C = m.hidden;
  auto add = [&](LayerKind k, std::optional<size_t> block, const std::string& label) -> Layer& {
    Layer l;
    l.idx = idx++; l.block_idx = block; l.kind = k; l.label = label; l.hidden = m.hidden; l.eps = m.rms_norm_eps;
    g.layers.push_back(l);
    return g.layers.back();
  };
  Layer& em = add(LayerKind::Embedding, std::nullopt, "embed_tokens");
  em.vocab = m.vocab;
  em.params.push_back({"embed", {m.vocab, C}, Dtype::Bf16});
  auto elems = [](const std::vector<Param>& ps) { uint64_t n = 0; for (auto& p : ps) n += p.numel(); return n; };
  for (size_t b = 0; b < layers.size(); ++b) {
    const Json& d = layers[b];
    const std::string type = d.at("type").as_string(), p = "l" + std::to_string(b) + ".";
    const bool q_latent = type == "latent_attention", gated = type == "latent_attention_2";
    if (!q_latent && !gated) throw ImportError("layer " + std::to_string(b) + ": mixer type `" + type + "` is not supported");
    const bool shared = d.has("weights_of") && !d.at("weights_of").is_null();
    const Json& mx = d.at("mixer");
    const uint64_t H = cfg_usize(mx, "heads"), D = cfg_usize(mx, "dim"), R = cfg_usize(mx, "rot_dim"), V = cfg_usize(mx, "vdim"), K = cfg_usize(mx, "kv_rank");
    std::vector<Param> ps;
    if (q_latent) {
      const uint64_t Q = cfg_usize(mx, "q_rank");
      ps.push_back({p + "mix.dq", {Q, C}, Dtype::Bf16});
      ps.push_back({p + "mix.dq.norm", {Q}, Dtype::Bf16});
      ps.push_back({p + "mix.uq", {H * (D + R), Q}, Dtype::Bf16});
    } else {
      ps.push_back({p + "mix.q", {H * (D + R), C}, Dtype::Bf16});
    }
    ps.push_back({p + "mix.dkv", {K + R, C}, Dtype::Bf16});
    ps.push_back({p + "mix.dkv.norm", {K}, Dtype::Bf16});
    ps.push_back({p + "mix.uk", {H * D, K}, Dtype::Bf16});
    ps.push_back({p + "mix.uv", {H * V, K}, Dtype::Bf16});
    if (gated) ps.push_back({p + "mix.g", {H * V, C}, Dtype::Bf16});
    ps.push_back({p + "mix.o", {C, H * V}, Dtype::Bf16});
    ps.push_back({p + "canon1", {C, taps}, Dtype::Bf16});
    {
      Layer& a = add(LayerKind::Attention, b, type);
      a.num_heads = H; a.num_kv_heads = 1; a.head_dim = D + R; a.kv_rank = K; a.rot_dim = R; a.v_dim = V; a.gated = gated;
      a.q_rank = q_latent ? cfg_usize(mx, "q_rank") : 0;
      a.conv_taps = taps;
      a.rope_theta = mx.at("rot").at("base").as_double();
      if (shared) a.shared_elems = elems(ps); else a.params = ps;
      m.rope_theta = a.rope_theta;
    }
    m.num_attention_heads = std::max<size_t>(m.num_attention_heads, H);
    m.head_dim = std::max<size_t>(m.head_dim, D + R);
    Layer& n1 = add(LayerKind::RmsNorm, b, "norm1");
    if (!shared) n1.params.push_back({p + "norm1", {}, Dtype::Bf16});
    if (!d.has("mlp") || d.at("mlp").is_null()) continue;
    const Json& ml = d.at("mlp");
    const std::string kind = ml.at("kind").as_string();
    ps.clear();
    if (kind == "dense") {
      const uint64_t F = cfg_usize(ml, "ff");
      ps.push_back({p + "mlp.up", {F, C}, Dtype::Bf16});
      ps.push_back({p + "mlp.down", {C, F}, Dtype::Bf16});
      ps.push_back({p + "mlp.act", {4}, Dtype::Bf16});
      Layer& f = add(LayerKind::Mlp, b, "mlp");
      f.intermediate = F;
      f.activation = "poly_norm";
      if (shared) f.shared_elems = elems(ps); else f.params = ps;
      m.intermediate = std::max<size_t>(m.intermediate, F);
    } else if (kind == "moe") {
      const uint64_t F = cfg_usize(ml.at("expert"), "ff"), E = cfg_usize(ml.at("router"), "experts");
      for (uint64_t e = 0; e < E; ++e) {
        const std::string q = p + "mlp.e" + std::to_string(e) + ".";
        ps.push_back({q + "gate", {F, C}, Dtype::Bf16});
        ps.push_back({q + "up", {F, C}, Dtype::Bf16});
        ps.push_back({q + "down", {C, F}, Dtype::Bf16});
      }
      ps.push_back({p + "mlp.router", {E, C}, Dtype::Bf16});
      Layer& f = add(LayerKind::Moe, b, "moe");
      f.intermediate = F; f.num_experts = E; f.top_k = cfg_usize(ml.at("router"), "top");
      f.activation = "clamped_glu";
      if (shared) f.shared_elems = elems(ps); else f.params = ps;
      m.intermediate = std::max<size_t>(m.intermediate, F * E);
    } else {
      throw ImportError("layer " + std::to_string(b) + ": feed-forward kind `" + kind + "` is not supported");
    }
    Layer& n2 = add(LayerKind::RmsNorm, b, "norm2");
    if (!shared) n2.params.push_back({p + "norm2", {}, Dtype::Bf16});
  }
  Layer& n = add(LayerKind::RmsNorm, std::nullopt, "norm");
  n.params.push_back({"final.norm", {}, Dtype::Bf16});
  Layer& l = add(LayerKind::Lmhead, std::nullopt, "lm_head");
  l.vocab = m.vocab;
  l.params.push_back({"head", {m.vocab, C}, Dtype::Bf16});
  g.meta = m;
  return g;
}

// The runs of a list of layers of which a range may run several times (`loop`).
struct LoopRuns {
  size_t start = 0, stop = 0, times = 1;
  bool looped = false;
  std::vector<std::pair<size_t, size_t>> runs;      // (layer, pass)
  bool opens(size_t layer) const { return looped && layer == start; }
};
inline LoopRuns read_loop(const Json& cfg, size_t n) {
  LoopRuns l;
  if (const Json* loop = cfg.find("loop"); loop && !loop->is_null()) {
    l.looped = true;
    l.start = cfg_usize(*loop, "start"); l.stop = cfg_usize(*loop, "stop"); l.times = cfg_usize(*loop, "times");
    if (l.start >= l.stop || l.stop > n || l.times < 1) throw ImportError("config.json: `loop` is not a range of the layers");
  }
  for (size_t i = 0; i < n;) {
    if (l.opens(i)) {
      for (size_t t = 0; t < l.times; ++t)
        for (size_t j = l.start; j < l.stop; ++j) l.runs.push_back({j, t});
      i = l.stop;
    } else {
      l.runs.push_back({i++, 0});
    }
  }
  return l;
}

// A design of parallel layers (Sikalorn): x <- x + (mixer(h) + ff(h)) with h = tanh(alpha x) w + b, and a range of layers that
// may run several times. One block per run; the runs after a layer's first own no parameters.
inline Graph import_parallel(const Json& cfg) {
  ModelMeta m;
  m.architecture = cfg.at("architecture").as_string();
  m.layered = m.parallel = true;
  m.hidden = cfg_usize(cfg, "width");
  m.vocab = cfg_usize(cfg, "vocab");
  m.max_position = cfg.has("max_position_embeddings") && !cfg.at("max_position_embeddings").is_null() ? cfg_usize(cfg, "max_position_embeddings") : 131072;
  for (const char* k : {"norm", "layers"})
    if (!cfg.has(k)) throw ImportError(std::string("config.json: missing `") + k + "`");
  m.rms_norm_eps = cfg.at("norm").at("eps").as_double();
  const auto& layers = cfg.at("layers").items();
  if (layers.empty()) throw ImportError("config.json: `layers` is empty");
  m.num_kv_heads = 1;
  const LoopRuns lr = read_loop(cfg, layers.size());
  const auto& runs = lr.runs;
  m.num_layers = runs.size();
  Graph g;
  size_t idx = 0;
  const uint64_t C = m.hidden;
  auto add = [&](LayerKind k, std::optional<size_t> block, const std::string& label) -> Layer& {
    Layer l;
    l.idx = idx++; l.block_idx = block; l.kind = k; l.label = label; l.hidden = m.hidden; l.eps = m.rms_norm_eps;
    g.layers.push_back(l);
    return g.layers.back();
  };
  auto elems = [](const std::vector<Param>& ps) { uint64_t n = 0; for (auto& p : ps) n += p.numel(); return n; };
  auto norm_params = [&](const std::string& n) {
    return std::vector<Param>{{n, {C}, Dtype::Bf16}, {n + ".b", {C}, Dtype::Bf16}, {n + ".alpha", {}, Dtype::Bf16}};
  };
  // parameters and cache / state sizes of the mixers
  auto window_attention = [&](const Json& mx, const std::string& p, Layer& a, std::vector<Param>& ps) {
    const uint64_t H = cfg_usize(mx, "heads"), K = cfg_usize(mx, "kv_heads"), D = cfg_usize(mx, "dim"), V = cfg_usize(mx, "vdim");
    ps.push_back({p + "q", {H * D, C}, Dtype::Bf16});
    ps.push_back({p + "k", {K * D, C}, Dtype::Bf16});
    ps.push_back({p + "v", {K * V, C}, Dtype::Bf16});
    ps.push_back({p + "q.norm", {H * D}, Dtype::Bf16});
    ps.push_back({p + "k.norm", {K * D}, Dtype::Bf16});
    ps.push_back({p + "o", {C, H * V}, Dtype::Bf16});
    a.num_heads = H; a.num_kv_heads = K; a.head_dim = D; a.v_dim = V; a.kv_elems = K * (D + V);
    if (const Json* w = mx.find("mask"); w && !w->is_null() && w->has("size") && !w->at("size").is_null()) a.window = cfg_usize(*w, "size");
    a.rope_theta = mx.at("rot").at("base").as_double();
    m.rope_theta = a.rope_theta;
    m.num_attention_heads = std::max<size_t>(m.num_attention_heads, H);
    m.head_dim = std::max<size_t>(m.head_dim, D);
  };
  auto recurrence = [&](const Json& mx, const std::string& kind, const std::string& p, Layer& a, std::vector<Param>& ps) {
    const uint64_t H = cfg_usize(mx, "heads"), V = cfg_usize(mx, "vdim"), D = cfg_usize(mx, kind == "ssd" ? "state" : "dim");
    const uint64_t G = kind == "ssd" ? cfg_usize(mx, "groups") : kind == "delta" ? cfg_usize(mx, "kv_heads") : H;
    const uint64_t taps = kind == "lightning" ? 1 : cfg_usize(mx, "conv"), channels = kind == "lightning" ? 0 : H * V + 2 * G * D;
    if (kind == "ssd") {
      ps.push_back({p + "in", {2 * H * V + 2 * G * D + H, C}, Dtype::Bf16});
      ps.push_back({p + "conv", {channels, taps}, Dtype::Bf16});
      ps.push_back({p + "conv.b", {channels}, Dtype::Bf16});
      for (const char* n : {"dt_bias", "A_log", "D"}) ps.push_back({p + n, {H}, Dtype::Bf16});
      ps.push_back({p + "norm", {H * V}, Dtype::Bf16});
    } else {
      const std::vector<std::pair<std::string, uint64_t>> qkv = {{"q", G * D}, {"k", G * D}, {"v", H * V}};
      for (auto& [n, rows] : qkv) ps.push_back({p + n, {rows, C}, Dtype::Bf16});
      ps.push_back({p + "g", {H * V, C}, Dtype::Bf16});
      if (kind == "delta") {
        for (const char* n : {"b", "a"}) ps.push_back({p + n, {H, C}, Dtype::Bf16});
        for (auto& [n, rows] : qkv) ps.push_back({p + n + ".conv", {rows, taps}, Dtype::Bf16});
        for (const char* n : {"A_log", "dt_bias"}) ps.push_back({p + n, {H}, Dtype::Bf16});
        ps.push_back({p + "norm", {V}, Dtype::Bf16});
      } else {
        ps.push_back({p + "norm", {H * V}, Dtype::Bf16});
      }
    }
    ps.push_back({p + "o", {C, H * V}, Dtype::Bf16});
    if (a.num_heads == 0) { a.num_heads = H; a.num_kv_heads = G; a.head_dim = D; a.v_dim = V; }
    m.num_attention_heads = std::max<size_t>(m.num_attention_heads, a.num_heads);
    m.head_dim = std::max<size_t>(m.head_dim, a.head_dim);
    a.conv_taps = taps;
    a.state_elems = H * D * V;
    a.state_bytes = 4 * a.state_elems + (taps > 1 ? 2 * taps * channels : 0);
  };
  Layer& em = add(LayerKind::Embedding, std::nullopt, "embed_tokens");
  em.vocab = m.vocab;
  em.params.push_back({"embed", {m.vocab, C}, Dtype::Bf16});
  for (size_t b = 0; b < runs.size(); ++b) {
    const auto [i, pass] = runs[b];
    const bool shared = pass > 0;
    const Json& d = layers[i];
    const std::string type = d.at("type").as_string(), p = "l" + std::to_string(i) + ".";
    {
      Layer& n1 = add(LayerKind::RmsNorm, b, "norm1");
      if (!shared) n1.params = norm_params(p + "norm1");
    }
    std::vector<Param> ps;
    Layer& a = add(LayerKind::Attention, b, type);
    a.parallel = true;
    const Json& mx = d.at("mixer");
    if (type == "parallel") {
      window_attention(mx.at("left"), p + "mix.left.", a, ps);
      recurrence(mx.at("right"), "ssd", p + "mix.right.", a, ps);
    } else if (type == "delta" || type == "lightning") {
      recurrence(mx, type, p + "mix.", a, ps);
    } else {
      throw ImportError("layer " + std::to_string(i) + ": mixer type `" + type + "` is not supported");
    }
    if (lr.opens(i)) {
      a.opens_pass = true;
      ps.push_back({"loop.in", {C, 2 * C}, Dtype::Bf16});
      ps.push_back({"loop.step", {lr.times, C}, Dtype::Bf16});
    }
    if (shared) a.shared_elems = elems(ps); else a.params = ps;
    if (!d.has("mlp") || d.at("mlp").is_null()) continue;
    const Json& ml = d.at("mlp");
    if (ml.at("kind").as_string() != "dense") throw ImportError("layer " + std::to_string(i) + ": feed-forward kind `" + ml.at("kind").as_string() + "` is not supported");
    const uint64_t F = cfg_usize(ml, "ff");
    ps = {{p + "mlp.up", {F, C}, Dtype::Bf16}, {p + "mlp.down", {C, F}, Dtype::Bf16}};
    Layer& f = add(LayerKind::Mlp, b, "mlp");
    f.intermediate = F;
    f.activation = "relu2";
    if (shared) f.shared_elems = elems(ps); else f.params = ps;
    m.intermediate = std::max<size_t>(m.intermediate, F);
  }
  Layer& n = add(LayerKind::RmsNorm, std::nullopt, "norm");
  n.params = norm_params("final.norm");
  Layer& l = add(LayerKind::Lmhead, std::nullopt, "lm_head");
  l.vocab = m.vocab;
  l.params.push_back({"head", {m.vocab, C}, Dtype::Bf16});
  g.meta = m;
  return g;
}

// A design of pre-norm layers with an fp32 stream. One block per run of a layer; the runs after a layer's first own no parameters.
//   Barorax   differential attention, attention inside chunks, selective scans; routed experts with one that runs for every token; a
//             range of layers that may run several times
//   Derusun   latent attention, attention over a window that keeps the first tokens, delta rules with a decay per key channel; clamped
//             gated units; a token shift in front of every mixer (the last normed row is part of a sequence's state) and an average over
//             depth behind every layer
inline Graph import_prenorm(const Json& cfg) {
  ModelMeta m;
  m.architecture = cfg.at("architecture").as_string();
  m.layered = m.prenorm = true;
  m.shifted = m.architecture == "Derusun";
  m.hidden = cfg_usize(cfg, "width");
  m.vocab = cfg_usize(cfg, "vocab");
  m.max_position = cfg.has("max_position_embeddings") && !cfg.at("max_position_embeddings").is_null() ? cfg_usize(cfg, "max_position_embeddings") : 131072;
  for (const char* k : {"norm", "layers"})
    if (!cfg.has(k)) throw ImportError(std::string("config.json: missing `") + k + "`");
  m.rms_norm_eps = cfg.at("norm").at("eps").as_double();
  const auto& layers = cfg.at("layers").items();
  if (layers.empty()) throw ImportError("config.json: `layers` is empty");
  m.num_kv_heads = 1;
  const LoopRuns lr = read_loop(cfg, layers.size());
  m.num_layers = lr.runs.size();
  Graph g;
  size_t idx = 0;
  const uint64_t C = m.hidden;
  auto add = [&](LayerKind k, std::optional<size_t> block, const std::string& label) -> Layer& {
    Layer l;
    l.idx = idx++; l.block_idx = block; l.kind = k; l.label = label; l.hidden = m.hidden; l.eps = m.rms_norm_eps;
    g.layers.push_back(l);
    return g.layers.back();
  };
  auto elems = [](const std::vector<Param>& ps) { uint64_t n = 0; for (auto& p : ps) n += p.numel(); return n; };
  Layer& em = add(LayerKind::Embedding, std::nullopt, "embed_tokens");
  em.vocab = m.vocab;
  em.params.push_back({"embed", {m.vocab, C}, Dtype::Bf16});
  for (size_t b = 0; b < lr.runs.size(); ++b) {
    const auto [i, pass] = lr.runs[b];
    const bool shared = pass > 0;
    const Json& d = layers[i];
    const std::string type = d.at("type").as_string(), p = "l" + std::to_string(i) + ".", q = p + "mix.";
    {
      Layer& n1 = add(LayerKind::RmsNorm, b, "norm1");
      if (!shared) n1.params.push_back({p + "norm1", {C}, Dtype::Bf16});
    }
    std::vector<Param> ps;
    Layer& a = add(LayerKind::Attention, b, type);
    a.parallel = true;
    const Json& mx = d.at("mixer");
    auto param = [&](const std::string& n, std::vector<uint64_t> shape) { ps.push_back({q + n, std::move(shape), Dtype::Bf16}); };
    auto heads = [&](uint64_t H, uint64_t K, uint64_t D, uint64_t V) {
      a.num_heads = H; a.num_kv_heads = K; a.head_dim = D; a.v_dim = V;
      m.num_attention_heads = std::max<size_t>(m.num_attention_heads, H);
      m.head_dim = std::max<size_t>(m.head_dim, D);
    };
    if (m.shifted) {
      const uint64_t H = cfg_usize(mx, "heads"), D = cfg_usize(mx, "dim"), V = cfg_usize(mx, "vdim");
      if (type == "latent_attention") {
        const uint64_t R = cfg_usize(mx, "rot_dim"), K = cfg_usize(mx, "kv_rank");
        param("q", {H * (D + R), C});
        param("dkv", {K + R, C});
        param("dkv.norm", {K});
        param("uk", {H * D, K});
        param("uv", {H * V, K});
        param("sink", {H});
        heads(H, 1, D, V);
        a.kv_rank = K; a.rot_dim = R; a.kv_elems = K + R;
        a.rope_theta = mx.at("rot").at("base").as_double();
        m.rope_theta = a.rope_theta;
      } else if (type == "attention") {
        const uint64_t K = cfg_usize(mx, "kv_heads");
        param("q", {H * D, C});
        param("k", {K * D, C});
        param("v", {K * V, C});
        param("q.b", {H * D});
        param("k.b", {K * D});
        param("v.b", {K * V});
        param("q.norm", {D});
        param("k.norm", {D});
        if (const Json* vm = mx.find("v_mix"); vm && !vm->is_null() && vm->as_bool()) param("vmix", {});
        param("sink", {H});
        heads(H, K, D, V);
        a.kv_elems = K * (D + V);
        if (const Json* w = mx.find("mask"); w && !w->is_null() && w->has("size") && !w->at("size").is_null() && cfg_usize(*w, "size") > 0)
          a.window = cfg_usize(*w, "size") + (w->has("keep_first") && !w->at("keep_first").is_null() ? cfg_usize(*w, "keep_first") : 0);
      } else if (type == "channel_delta") {
        const uint64_t G = cfg_usize(mx, "kv_heads"), taps = cfg_usize(mx, "conv"), channels = H * V + 2 * G * D;
        auto rank = [&](const char* n) { return mx.has(n) && !mx.at(n).is_null() ? (uint64_t)cfg_usize(mx, n) : D; };
        const uint64_t RA = rank("decay_rank"), RG = rank("gate_rank");
        param("q", {G * D, C});
        param("k", {G * D, C});
        param("v", {H * V, C});
        param("b", {H, C});
        param("a1", {RA, C});
        param("g1", {RG, C});
        param("q.conv", {G * D, taps});
        param("k.conv", {G * D, taps});
        param("v.conv", {H * V, taps});
        param("A_log", {H});
        param("norm", {V});
        param("a2", {H * D, RA});
        param("dt_bias", {H * D});
        param("g2", {H * V, RG});
        heads(H, G, D, V);
        a.bottlenecks = true;
        a.conv_taps = taps;
        a.state_elems = H * D * V;
        a.state_bytes = 4 * a.state_elems + (taps > 1 ? 2 * taps * channels : 0);
      } else {
        throw ImportError("layer " + std::to_string(i) + ": mixer type `" + type + "` is not supported");
      }
      param("o", {C, H * V});
      ps.push_back({p + "shift", {C}, Dtype::Bf16});
      ps.push_back({p + "dwa", {i + 2}, Dtype::Bf16});
      a.state_bytes += 4 * C;
    } else if (type == "attention" || type == "attention_2") {
      const bool differential = type == "attention";
      const uint64_t H = cfg_usize(mx, "heads"), K = cfg_usize(mx, "kv_heads"), D = cfg_usize(mx, "dim"), V = cfg_usize(mx, "vdim"), M = differential ? 2 : 1;
      param("q", {H * M * D, C});
      param("k", {K * M * D, C});
      param("v", {K * V, C});
      if (differential) {
        for (const char* n : {"lq1", "lk1", "lq2", "lk2"}) param(n, {D});
        param("g", {H * V, C});
      } else {
        a.window = cfg_usize(mx.at("mask"), "size");     // a row sees at most its chunk
      }
      param("o", {C, H * V});
      a.num_heads = H * M; a.num_kv_heads = K; a.head_dim = D; a.v_dim = V; a.kv_elems = K * (M * D + V); a.gated = differential;
      a.rope_theta = mx.at("rot").at("base").as_double();
      m.rope_theta = a.rope_theta;
      m.num_attention_heads = std::max<size_t>(m.num_attention_heads, H);
      m.head_dim = std::max<size_t>(m.head_dim, D);
    } else if (type == "mamba1") {
      const uint64_t I = cfg_usize(mx, "inner"), N = cfg_usize(mx, "state"), R = cfg_usize(mx, "dt_rank"), taps = cfg_usize(mx, "conv");
      param("in", {2 * I, C});
      param("conv", {I, taps});
      param("conv.b", {I});
      param("x", {R + 2 * N, I});
      param("dt", {I, R});
      param("dt.b", {I});
      param("A_log", {I, N});
      param("D", {I});
      param("o", {C, I});
      a.selective = true;
      a.num_heads = a.num_kv_heads = 1; a.head_dim = N; a.v_dim = I;
      a.conv_taps = taps;
      a.state_elems = I * N;
      a.state_bytes = 4 * I * N + (taps > 1 ? 2 * taps * I : 0);
      m.num_attention_heads = std::max<size_t>(m.num_attention_heads, 1);
      m.head_dim = std::max<size_t>(m.head_dim, N);
    } else {
      throw ImportError("layer " + std::to_string(i) + ": mixer type `" + type + "` is not supported");
    }
    if (lr.opens(i)) {
      a.opens_pass = true;
      ps.push_back({"loop.step", {lr.times, C}, Dtype::Bf16});
    }
    if (shared) a.shared_elems = elems(ps); else a.params = ps;
    if (!d.has("mlp") || d.at("mlp").is_null()) continue;
    const Json& ml = d.at("mlp");
    if (ml.at("kind").as_string() != (m.shifted ? "dense" : "moe"))
      throw ImportError("layer " + std::to_string(i) + ": feed-forward kind `" + ml.at("kind").as_string() + "` is not supported");
    {
      Layer& n2 = add(LayerKind::RmsNorm, b, "norm2");
      if (!shared) n2.params.push_back({p + "norm2", {C}, Dtype::Bf16});
    }
    if (m.shifted) {
      const uint64_t F = cfg_usize(ml, "ff");
      Layer& f = add(LayerKind::Mlp, b, "mlp");
      f.intermediate = F;
      f.activation = "clamped_glu";
      f.params = {{p + "mlp.gate", {F, C}, Dtype::Bf16}, {p + "mlp.up", {F, C}, Dtype::Bf16}, {p + "mlp.down", {C, F}, Dtype::Bf16}};
      m.intermediate = std::max<size_t>(m.intermediate, F);
      continue;
    }
    const uint64_t F = cfg_usize(ml.at("expert"), "ff"), E = cfg_usize(ml.at("router"), "experts");
    ps.clear();
    auto expert = [&](const std::string& n, uint64_t ff) {
      ps.push_back({n + "gate", {ff, C}, Dtype::Bf16});
      ps.push_back({n + "up", {ff, C}, Dtype::Bf16});
      ps.push_back({n + "down", {C, ff}, Dtype::Bf16});
    };
    for (uint64_t e = 0; e < E; ++e) expert(p + "mlp.e" + std::to_string(e) + ".", F);
    ps.push_back({p + "mlp.router", {E, C}, Dtype::Bf16});
    Layer& f = add(LayerKind::Moe, b, "moe");
    if (ml.has("shared") && !ml.at("shared").is_null()) {
      f.always_ff = cfg_usize(ml.at("shared"), "ff");
      expert(p + "mlp.shared.", f.always_ff);
    }
    f.intermediate = F; f.num_experts = E; f.top_k = cfg_usize(ml.at("router"), "top");
    if (shared) f.shared_elems = elems(ps); else f.params = ps;
    m.intermediate = std::max<size_t>(m.intermediate, F * E);
  }
  Layer& n = add(LayerKind::RmsNorm, std::nullopt, "norm");
  n.params.push_back({"final.norm", {C}, Dtype::Bf16});
  Layer& l = add(LayerKind::Lmhead, std::nullopt, "lm_head");
  l.vocab = m.vocab;
  l.params.push_back({"head", {m.vocab, C}, Dtype::Bf16});
  g.meta = m;
  return g;
}

inline Graph import_model(const Json& cfg) {
  if (const Json* a = cfg.find("architecture"); a && !a->is_null()) {
    if (a->as_string() == "Zarorax") return import_layered(cfg);
    if (a->as_string() == "Sikalorn") return import_parallel(cfg);
    if (a->as_string() == "Barorax" || a->as_string() == "Derusun") return import_prenorm(cfg);
  }
  const Json* archs = cfg.find("architectures");
  if (!archs || !archs->is_array() || archs->size() == 0) throw ImportError("config.json: `architectures` is missing or empty");
  const std::string arch = archs->items()[0].as_string();
  const bool moe = arch == "MixtralForCausalLM";
  const bool dense = arch == "LlamaForCausalLM" || arch == "MistralForCausalLM" || arch == "Qwen2ForCausalLM";
  if (!moe && !dense) throw ImportError("architecture `" + arch + "` is not supported");
  if (const Json* act = cfg.find("hidden_act"); act && !act->is_null() && act->as_string() != "silu")
    throw ImportError("hidden_act `" + act->as_string() + "` is not supported (only silu)");

  ModelMeta m;
  m.architecture = arch;
  m.hidden = cfg_usize(cfg, "hidden_size");
  m.intermediate = cfg_usize(cfg, "intermediate_size");
  m.num_layers = cfg_usize(cfg, "num_hidden_layers");
  m.num_attention_heads = cfg_usize(cfg, "num_attention_heads");
  m.num_kv_heads = cfg.has("num_key_value_heads") && !cfg.at("num_key_value_heads").is_null()
                       ? cfg_usize(cfg, "num_key_value_heads") : m.num_attention_heads;
  m.vocab = cfg_usize(cfg, "vocab_size");
  m.max_position = cfg.has("max_position_embeddings") ? cfg_usize(cfg, "max_position_embeddings") : 8192;
  if (m.num_attention_heads == 0 || m.num_kv_heads == 0) throw ImportError("head counts must be positive");
  if (const Json* hd = cfg.find("head_dim"); hd && !hd->is_null()) m.head_dim = (size_t)hd->as_int();
  else {
    if (m.hidden % m.num_attention_heads) throw ImportError("hidden_size is not divisible by num_attention_heads and head_dim is absent");
    m.head_dim = m.hidden / m.num_attention_heads;
  }
  if (m.num_attention_heads % m.num_kv_heads) throw ImportError("num_attention_heads must be a multiple of num_key_value_heads (GQA)");
  // newer checkpoints nest theta and the frequency-scaling scheme in `rope_parameters`
  const Json* rp = cfg.find("rope_parameters");
  if (rp && (rp->is_null() || !rp->is_object())) rp = nullptr;
  m.rope_theta = cfg.has("rope_theta") && !cfg.at("rope_theta").is_null() ? cfg.at("rope_theta").as_double()
                 : (rp && rp->has("rope_theta") ? rp->at("rope_theta").as_double() : 1e4);
  {
    const Json* sc = cfg.find("rope_scaling");
    if (!sc || sc->is_null()) sc = rp;
    if (sc && sc->is_object()) {
      std::string kind = "default";
      if (const Json* t = sc->find("rope_type"); t && !t->is_null()) kind = t->as_string();
      else if (const Json* t2 = sc->find("type"); t2 && !t2->is_null()) kind = t2->as_string();
      if (kind != "default" && kind != "linear" && kind != "llama3")
        throw ImportError("rope scaling `" + kind + "` is not supported (plain, linear and llama3 are)");
    }
  }
  if (const Json* mb = cfg.find("mlp_bias"); mb && !mb->is_null() && mb->as_bool()) throw ImportError("mlp_bias = true is not supported");
  m.rms_norm_eps = cfg.has("rms_norm_eps") ? cfg.at("rms_norm_eps").as_double() : 1e-5;
  if (const Json* sw = cfg.find("sliding_window"); sw && !sw->is_null()) {
    const Json* use = cfg.find("use_sliding_window");
    // Qwen2 lists a window but applies it only with use_sliding_window. Where a window applies it becomes the position limit:
    // the kernels attend over the whole context, the same function up to that length.
    if (arch != "Qwen2ForCausalLM" || (use && !use->is_null() && use->as_bool())) {
      m.sliding_window = (size_t)sw->as_int();
      if (*m.sliding_window > 0 && *m.sliding_window < m.max_position) m.max_position = *m.sliding_window;
    }
  }
  m.tied_embeddings = cfg.has("tie_word_embeddings") && cfg.at("tie_word_embeddings").as_bool();
  // Qwen2 adds a bias to the q / k / v projections (none on o_proj). The Llama-style `attention_bias` switch adds one to
  // o_proj as well, which the runtime does not carry.
  m.qkv_bias = arch == "Qwen2ForCausalLM";
  if (const Json* ab = cfg.find("attention_bias"); ab && !ab->is_null() && ab->as_bool() && !m.qkv_bias)
    throw ImportError("attention_bias = true (biases on q, k, v and o_proj) is not supported for " + arch);
  if (moe) {
    m.num_experts = cfg_usize(cfg, "num_local_experts");
    m.top_k = cfg_usize(cfg, "num_experts_per_tok");
    if (*m.num_experts == 0 || *m.top_k == 0 || *m.top_k > *m.num_experts)
      throw ImportError("num_experts_per_tok must be in [1, num_local_experts]");
  }

  Graph g;
  g.meta = m;
  const uint64_t H = m.hidden, I = m.intermediate, D = m.head_dim, V = m.vocab;
  const uint64_t QO = m.num_attention_heads * D, KV = m.num_kv_heads * D;
  size_t idx = 0;
  auto add = [&](LayerKind k, std::optional<size_t> block, const std::string& label) -> Layer& {
    Layer l;
    l.idx = idx++; l.block_idx = block; l.kind = k; l.label = label;
    g.layers.push_back(l);
    return g.layers.back();
  };
  {
    Layer& e = add(LayerKind::Embedding, std::nullopt, "embed_tokens");
    e.vocab = V; e.hidden = H;
    e.params.push_back({"model.embed_tokens.weight", {V, H}, Dtype::Bf16});
  }
  for (size_t b = 0; b < m.num_layers; ++b) {
    const std::string pre = "model.layers." + std::to_string(b) + ".";
    Layer& n1 = add(LayerKind::RmsNorm, b, "input_layernorm");
    n1.hidden = H; n1.eps = m.rms_norm_eps;
    n1.params.push_back({pre + "input_layernorm.weight", {H}, Dtype::Bf16});
    Layer& a = add(LayerKind::Attention, b, "self_attn");
    a.num_heads = m.num_attention_heads; a.num_kv_heads = m.num_kv_heads; a.head_dim = D; a.hidden = H; a.rope_theta = m.rope_theta;
    a.params.push_back({pre + "self_attn.q_proj.weight", {QO, H}, Dtype::Bf16});
    a.params.push_back({pre + "self_attn.k_proj.weight", {KV, H}, Dtype::Bf16});
    a.params.push_back({pre + "self_attn.v_proj.weight", {KV, H}, Dtype::Bf16});
    a.params.push_back({pre + "self_attn.o_proj.weight", {H, QO}, Dtype::Bf16});
    if (m.qkv_bias) {
      a.params.push_back({pre + "self_attn.q_proj.bias", {QO}, Dtype::Bf16});
      a.params.push_back({pre + "self_attn.k_proj.bias", {KV}, Dtype::Bf16});
      a.params.push_back({pre + "self_attn.v_proj.bias", {KV}, Dtype::Bf16});
    }
    Layer& n2 = add(LayerKind::RmsNorm, b, "post_attention_layernorm");
    n2.hidden = H; n2.eps = m.rms_norm_eps;
    n2.params.push_back({pre + "post_attention_layernorm.weight", {H}, Dtype::Bf16});
    if (moe) {
      Layer& f = add(LayerKind::Moe, b, "block_sparse_moe");
      f.num_experts = *m.num_experts; f.top_k = *m.top_k; f.hidden = H; f.intermediate = I;
      f.params.push_back({pre + "block_sparse_moe.gate.weight", {(uint64_t)*m.num_experts, H}, Dtype::Bf16});
      for (size_t e = 0; e < *m.num_experts; ++e) {
        const std::string ep = pre + "block_sparse_moe.experts." + std::to_string(e) + ".";
        f.params.push_back({ep + "w1.weight", {I, H}, Dtype::Bf16});
        f.params.push_back({ep + "w2.weight", {H, I}, Dtype::Bf16});
        f.params.push_back({ep + "w3.weight", {I, H}, Dtype::Bf16});
      }
    } else {
      Layer& f = add(LayerKind::Mlp, b, "mlp");
      f.hidden = H; f.intermediate = I;
      f.params.push_back({pre + "mlp.gate_proj.weight", {I, H}, Dtype::Bf16});
      f.params.push_back({pre + "mlp.up_proj.weight", {I, H}, Dtype::Bf16});
      f.params.push_back({pre + "mlp.down_proj.weight", {H, I}, Dtype::Bf16});
    }
  }
  {
    Layer& n = add(LayerKind::RmsNorm, std::nullopt, "norm");
    n.hidden = H; n.eps = m.rms_norm_eps;
    n.params.push_back({"model.norm.weight", {H}, Dtype::Bf16});
    Layer& l = add(LayerKind::Lmhead, std::nullopt, "lm_head");
    l.vocab = V; l.hidden = H; l.tied = m.tied_embeddings;
    if (!m.tied_embeddings) l.params.push_back({"lm_head.weight", {V, H}, Dtype::Bf16});
  }
  return g;
}

inline Graph import_model_str(const std::string& text) {
  try {
    return import_model(Json::parse(text));
  } catch (const JsonError& e) {
    throw ImportError(std::string("config.json: ") + e.what());
  }
}

}  // namespace skein
