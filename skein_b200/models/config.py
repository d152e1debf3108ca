"""Model and parallel-layout descriptions used by the decoder graph.

ModelConfig is read from a HuggingFace ``config.json`` (MixtralForCausalLM, LlamaForCausalLM and
the Llama-shaped Mistral / Qwen2 families), or from the configuration of a design that lists its layers one by one
(models/layered.py). The reference imports Mixtral only
(crates/skein_ir/src/model/mod.rs:33-47, model/mixtral.rs:74-372) and rejects the rest; here the
dense Llama-style block is a Mixtral block with a plain SwiGLU MLP instead of routed experts.
"""
from __future__ import annotations

import json
from dataclasses import asdict, dataclass
from pathlib import Path

from .layered import LAYERED_ARCHS, PARALLEL_ARCHS, PRENORM_ARCHS, SHIFTED_ARCHS, DenseFFSpec, RoutedFFSpec, SpecError, layers_to_list, param_shapes, parse_layers, unroll_loop
from .parallel_layers import attention_of, parse_loop, recurrence_of
from .prenorm_layers import fill_ranks

MOE_ARCHS = {"MixtralForCausalLM"}
DENSE_ARCHS = {"LlamaForCausalLM", "MistralForCausalLM", "Qwen2ForCausalLM"}


class ImportError_(ValueError):
    """A config.json that cannot be turned into a consistent model."""


@dataclass
class ModelConfig:
    architecture: str = "MixtralForCausalLM"
    hidden_size: int = 4096
    intermediate_size: int = 14336
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    vocab_size: int = 32000
    rms_norm_eps: float = 1e-5
    rope_theta: float = 1e6
    num_experts: int = 8          # 0 = dense MLP
    top_k: int = 2
    max_position_embeddings: int = 32768
    tie_word_embeddings: bool = False
    name: str = "mixtral-8x7b"
    qkv_bias: bool = False        # the q / k / v projections carry a bias each (Qwen2)
    eos_token_id: int = -1        # token that ends a generation (-1: none known)
    rope_scaling: dict | None = None   # the checkpoint's RoPE frequency scaling ("linear" or "llama3"), None = plain RoPE
    # designs that list their layers (models/layered.py): per-layer specifications, () for the uniform families
    layers: tuple = ()
    conv_taps: int = 0            # taps of the input convolution
    post_alpha: float = 1.0       # weight of the residual inside the post-norms
    loop: tuple | None = None     # (start, stop, times): checkpoint layers that run several times (`layers` lists every run)
    norm_groups: int = 1          # equal parts of a normed row that have a root mean square each

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_layered(self) -> bool:
        return bool(self.layers)

    @property
    def is_parallel(self) -> bool:
        """Layers are x + mixer(h) + ff(h) (models/parallel_layers.py)."""
        return self.architecture in PARALLEL_ARCHS

    @property
    def is_prenorm(self) -> bool:
        """Layers are x + mixer(norm1(x)), x + ff(norm2(x)) with an fp32 stream (models/prenorm_layers.py)."""
        return self.architecture in PRENORM_ARCHS

    @property
    def is_shifted(self) -> bool:
        """Pre-norm layers whose mixer also reads the previous token's row, and whose stream is averaged over depth."""
        return self.architecture in SHIFTED_ARCHS

    @property
    def has_state(self) -> bool:
        """Sequences carry a recurrent state (or the last token's rows) beside their cache pages: each needs a state slot, and a prefix of
        cached pages alone does not bring a sequence back."""
        return self.is_shifted or any(recurrence_of(l.mixer) is not None for l in self.layers)

    def state_bytes_per_slot(self, elem: int = 2) -> int:
        rows = 4 * self.hidden_size * self.num_layers if self.is_shifted else 0
        return rows + sum(recurrence_of(l.mixer).state_bytes(elem) for l in self.layers if recurrence_of(l.mixer) is not None)

    @property
    def default_page_size(self) -> int:
        """Tokens per cache page: a latent cache row is small and one per token, so its pages are larger."""
        return 64 if self.is_layered else 16

    def cache_bytes_per_page(self, page_size: int, tp: int = 1, blocks=None, elem: int = 2) -> int:
        """Bytes of one page over the listed blocks (default: all) on one rank."""
        blocks = range(self.num_layers) if blocks is None else blocks
        if not self.is_layered:
            return 2 * (self.num_kv_heads // tp) * page_size * self.head_dim * elem * len(blocks)
        tail = self.conv_tail_rows(page_size) * self.hidden_size
        return sum((self.layers[b].mixer.cache_elems_per_token * page_size + tail) * elem for b in blocks)

    def conv_tail_rows(self, page_size: int) -> int:
        """Rows per cache page that keep the input convolution's last inputs. One more than the taps that look back, so that a
        step writes no row it reads: running a step twice (a graph's warm-up before its capture) gives the same result twice."""
        return min(self.conv_taps, page_size) if self.conv_taps > 1 else 0

    def param_shapes(self) -> dict:
        """Checkpoint tensor name -> shape (designs that list their layers)."""
        return param_shapes(self)

    def validate(self) -> None:
        if self.is_layered:
            if self.conv_taps < 1 and not (self.is_parallel or self.is_prenorm):
                raise ImportError_("canon.taps must be at least 1")
            if self.norm_groups < 1 or self.hidden_size % self.norm_groups:
                raise ImportError_("norm.groups must divide width")
            return
        if self.num_heads % self.num_kv_heads != 0:
            raise ImportError_("num_attention_heads must be a multiple of num_key_value_heads")
        if self.is_moe and not (1 <= self.top_k <= self.num_experts):
            raise ImportError_("num_experts_per_tok must be in [1, num_local_experts]")
        if self.head_dim % 2 != 0:
            raise ImportError_("head_dim must be even (RoPE rotates pairs)")

    def param_count(self) -> int:
        if self.is_layered:
            total = 0
            for shape in self.param_shapes().values():
                n = 1
                for d in shape:
                    n *= d
                total += n
            return total
        H, I, D = self.hidden_size, self.intermediate_size, self.head_dim
        attn = H * (self.num_heads * D) * 2 + H * (self.num_kv_heads * D) * 2
        if self.qkv_bias:
            attn += (self.num_heads + 2 * self.num_kv_heads) * D
        ffn = 3 * H * I * max(self.num_experts, 1) + (H * self.num_experts if self.is_moe else 0)
        per_block = attn + ffn + 2 * H
        emb = self.vocab_size * H
        return self.num_layers * per_block + emb + H + (0 if self.tie_word_embeddings else emb)

    def to_dict(self) -> dict:
        return asdict(self)

    @staticmethod
    def from_hf_dict(d: dict, name: str | None = None) -> "ModelConfig":
        if d.get("architecture") in LAYERED_ARCHS:
            return ModelConfig._from_layered_dict(d, name)
        archs = d.get("architectures") or []
        if not archs:
            raise ImportError_("config.json has no `architectures`")
        arch = archs[0]
        if arch not in MOE_ARCHS | DENSE_ARCHS:
            raise ImportError_(f"architecture {arch} is not supported")
        act = d.get("hidden_act", "silu")
        if act != "silu":
            raise ImportError_(f"hidden_act {act!r} is not supported (only silu)")
        H = int(d["hidden_size"])
        nh = int(d["num_attention_heads"])
        hd = d.get("head_dim") or (H // nh)
        if d.get("head_dim") is None and H % nh != 0:
            raise ImportError_("hidden_size is not divisible by num_attention_heads and head_dim is absent")
        # newer checkpoints nest theta and the scaling scheme in `rope_parameters`; older ones have `rope_theta` and
        # `rope_scaling` at the top level
        rp = d.get("rope_parameters") or {}
        theta = d.get("rope_theta", rp.get("rope_theta", 1e4))
        scaling = d.get("rope_scaling") or ({k: v for k, v in rp.items() if k != "rope_theta"} if rp else None)
        kind = (scaling or {}).get("rope_type") or (scaling or {}).get("type") or "default"
        if kind == "default":
            scaling = None
        elif kind not in ("linear", "llama3"):
            raise ImportError_(f"rope scaling {kind!r} is not supported (plain, linear and llama3 are)")
        if float(d.get("partial_rotary_factor", rp.get("partial_rotary_factor", 1.0)) or 1.0) != 1.0:
            raise ImportError_("partial rotary embeddings are not supported")
        if d.get("mlp_bias"):
            raise ImportError_("mlp_bias = true is not supported")
        cfg = ModelConfig(
            architecture=arch, hidden_size=H, intermediate_size=int(d["intermediate_size"]),
            num_layers=int(d["num_hidden_layers"]), num_heads=nh,
            num_kv_heads=int(d.get("num_key_value_heads", nh)), head_dim=int(hd), vocab_size=int(d["vocab_size"]),
            rms_norm_eps=float(d.get("rms_norm_eps", 1e-5)), rope_theta=float(theta),
            num_experts=int(d.get("num_local_experts", 0)) if arch in MOE_ARCHS else 0,
            top_k=int(d.get("num_experts_per_tok", 0)) if arch in MOE_ARCHS else 0,
            max_position_embeddings=int(d.get("max_position_embeddings", 8192)),
            tie_word_embeddings=bool(d.get("tie_word_embeddings", False)),
            name=name or d.get("_name_or_path") or d.get("model_type", "model"),
            qkv_bias=arch == "Qwen2ForCausalLM", rope_scaling=dict(scaling) if scaling else None)
        eos = d.get("eos_token_id")
        if isinstance(eos, (list, tuple)):      # several end tokens: the engine stops on one, the first listed
            eos = eos[0] if eos else None
        cfg.eos_token_id = int(eos) if eos is not None else -1
        # Sliding-window attention (Mistral v0.1; Qwen2 only with use_sliding_window): the attention kernels attend over the
        # whole context, which is the same function as long as a sequence is no longer than the window, so the window
        # becomes the position limit and longer requests are refused instead of being answered differently.
        sw = d.get("sliding_window")
        if sw and (arch != "Qwen2ForCausalLM" or d.get("use_sliding_window")) and int(sw) < cfg.max_position_embeddings:
            cfg.max_position_embeddings = int(sw)
        if d.get("attention_bias") and not cfg.qkv_bias:
            raise ImportError_(f"attention_bias = true (biases on q, k, v and o_proj) is not supported for {arch}")
        cfg.validate()
        return cfg

    @staticmethod
    def _from_layered_dict(d: dict, name: str | None) -> "ModelConfig":
        try:
            arch = d["architecture"]
            layers = parse_layers(arch, d["layers"], d.get("loop"))
            if arch in PARALLEL_ARCHS | PRENORM_ARCHS:
                only = {"loop": parse_loop(d.get("loop"), len(d["layers"]))}
            else:
                only = {"taps": int(d["canon"]["taps"]), "alpha": float(d["postln_alpha"])}
            if arch in SHIFTED_ARCHS:
                only["groups"] = int(d["norm"].get("groups") or 1)
            cfg = ModelConfig.layered(arch, layers, width=int(d["width"]), vocab=int(d["vocab"]), eps=float(d["norm"]["eps"]),
                                      name=name or arch.lower(), **only)
        except KeyError as e:
            raise ImportError_(f"config.json: missing {e.args[0]!r}") from e
        except SpecError as e:
            raise ImportError_(str(e)) from e
        if not layers:
            raise ImportError_("config.json: `layers` is empty")
        cfg.max_position_embeddings = int(d.get("max_position_embeddings", cfg.max_position_embeddings))
        eos = d.get("eos_token_id")
        cfg.eos_token_id = int(eos) if eos is not None else -1
        return cfg

    @staticmethod
    def layered(arch: str, layers, width: int, vocab: int, taps: int = 0, alpha: float = 1.0, eps: float = 1e-5, max_pos: int = 131072,
                name: str = "layered", loop: tuple | None = None, groups: int = 1) -> "ModelConfig":
        """Configuration of a design that lists its layers. The single-valued fields describe its largest layer (planning and
        display only; the layer specifications decide what runs). The design sets no position limit: max_pos is the engine's.
        `loop` (start, stop, times): `layers` are its runs (models/layered.py: unroll_loop)."""
        ff = [l.mlp.ff * (l.mlp.experts if isinstance(l.mlp, RoutedFFSpec) else 1) for l in layers if l.mlp is not None]
        bases = [b for b in (getattr(attention_of(l.mixer) or l.mixer, "rope_base", None) for l in layers) if b is not None]
        cfg = ModelConfig(architecture=arch, hidden_size=width, intermediate_size=max(ff, default=0), num_layers=len(layers),
                          num_heads=max(l.mixer.heads for l in layers) if layers else 0, num_kv_heads=1,
                          head_dim=max(l.mixer.head_size for l in layers) if layers else 0, vocab_size=vocab,
                          rms_norm_eps=eps, rope_theta=bases[0] if bases else 1e4, num_experts=0, top_k=0,
                          max_position_embeddings=max_pos, name=name, layers=tuple(layers), conv_taps=taps, post_alpha=alpha, loop=loop, norm_groups=groups)
        cfg.validate()
        return cfg

    def to_hf_dict(self) -> dict:
        """The config.json fields that describe this model (what the planner and the lowering read)."""
        if self.is_parallel or self.is_prenorm:
            d = {"architecture": self.architecture, "width": self.hidden_size, "vocab": self.vocab_size, "norm": {"eps": self.rms_norm_eps},
                 "layers": layers_to_list(self.layers), "max_position_embeddings": self.max_position_embeddings}
            if self.is_shifted:
                d["norm"]["groups"] = self.norm_groups
            if self.loop is not None:
                d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
            return d
        if self.is_layered:
            return {"architecture": self.architecture, "width": self.hidden_size, "vocab": self.vocab_size, "norm": {"eps": self.rms_norm_eps},
                    "canon": {"taps": self.conv_taps}, "postln_alpha": self.post_alpha, "layers": layers_to_list(self.layers),
                    "max_position_embeddings": self.max_position_embeddings}
        d = {"architectures": [self.architecture], "hidden_size": self.hidden_size, "intermediate_size": self.intermediate_size,
             "num_hidden_layers": self.num_layers, "num_attention_heads": self.num_heads, "num_key_value_heads": self.num_kv_heads,
             "head_dim": self.head_dim, "vocab_size": self.vocab_size, "rms_norm_eps": self.rms_norm_eps, "rope_theta": self.rope_theta,
             "max_position_embeddings": self.max_position_embeddings, "tie_word_embeddings": self.tie_word_embeddings,
             "hidden_act": "silu"}
        if self.is_moe:
            d.update(num_local_experts=self.num_experts, num_experts_per_tok=self.top_k)
        if self.rope_scaling:
            d["rope_scaling"] = dict(self.rope_scaling)
        return d

    @staticmethod
    def from_file(path) -> "ModelConfig":
        p = Path(path)
        return ModelConfig.from_hf_dict(json.loads(sized_config(p.read_text(), p.parent)), name=p.stem.replace("_config", ""))


def checkpoint_shapes(path) -> dict:
    """Tensor name -> shape of a checkpoint (a safetensors file, or a directory with one or with shards), from the files' headers; empty
    where there is none."""
    p = Path(path)
    index = p / "model.safetensors.index.json"
    files = [p] if p.is_file() else sorted({p / f for f in json.loads(index.read_text())["weight_map"].values()}) if index.exists() \
        else [p / "model.safetensors"]
    shapes = {}
    for f in files:
        if f.suffix != ".safetensors" or not f.exists():
            continue
        with open(f, "rb") as fh:
            header = json.loads(fh.read(int.from_bytes(fh.read(8), "little")))
        shapes.update({n: tuple(t["shape"]) for n, t in header.items() if n != "__metadata__"})
    return shapes


def sized_config(config_json: str, checkpoint) -> str:
    """The configuration with the sizes that its design leaves to the checkpoint's tensors filled in (where there is a checkpoint)."""
    d = json.loads(config_json)
    if d.get("architecture") not in SHIFTED_ARCHS or checkpoint is None or not isinstance(d.get("layers"), list):
        return config_json
    shapes = checkpoint_shapes(checkpoint)
    return json.dumps(fill_ranks(d, shapes.get)) if shapes else config_json


def mixtral_8x7b() -> ModelConfig:
    return ModelConfig()


def mixtral_8x22b() -> ModelConfig:
    return ModelConfig(hidden_size=6144, intermediate_size=16384, num_layers=56, num_heads=48, num_kv_heads=8,
                       head_dim=128, vocab_size=32768, rope_theta=1e6, num_experts=8, top_k=2,
                       max_position_embeddings=65536, name="mixtral-8x22b")


def llama3_70b() -> ModelConfig:
    return ModelConfig(architecture="LlamaForCausalLM", hidden_size=8192, intermediate_size=28672, num_layers=80,
                       num_heads=64, num_kv_heads=8, head_dim=128, vocab_size=128256, rms_norm_eps=1e-5,
                       rope_theta=5e5, num_experts=0, top_k=0, max_position_embeddings=8192, name="llama3-70b")


def tiny_mixtral(layers=2, hidden=256, inter=512, heads=4, kv_heads=2, experts=4, vocab=512) -> ModelConfig:
    """A small Mixtral-shaped model for tests (head_dim stays 128: the attention kernels require it)."""
    return ModelConfig(hidden_size=hidden, intermediate_size=inter, num_layers=layers, num_heads=heads,
                       num_kv_heads=kv_heads, head_dim=128, vocab_size=vocab, num_experts=experts, top_k=2,
                       max_position_embeddings=4096, name="tiny-mixtral")


def tiny_llama(layers=2, hidden=256, inter=512, heads=4, kv_heads=2, vocab=512) -> ModelConfig:
    return ModelConfig(architecture="LlamaForCausalLM", hidden_size=hidden, intermediate_size=inter,
                       num_layers=layers, num_heads=heads, num_kv_heads=kv_heads, head_dim=128, vocab_size=vocab,
                       rope_theta=5e5, num_experts=0, top_k=0, max_position_embeddings=4096, name="tiny-llama")


def tiny_zarorax(width=192, vocab=384, taps=4, alpha=2.5, eps=1e-5) -> ModelConfig:
    """A small model of the Zarorax design for tests: both mixers, both feed-forwards, one shared layer, one without any."""
    from .layered import LatentMixerSpec, LayerSpec
    a = LatentMixerSpec("latent_attention_2", heads=3, dim=48, rot_dim=16, vdim=40, kv_rank=80, rope_base=1e4, scale=0.11, gated=True)
    b = LatentMixerSpec("latent_attention", heads=5, dim=24, rot_dim=32, vdim=32, kv_rank=96, rope_base=5e3, scale=0.13, q_rank=56)
    moe = RoutedFFSpec(ff=72, limit=1.5, experts=8, top=2, groups=4, keep=2)
    return ModelConfig.layered("Zarorax", (LayerSpec(a, DenseFFSpec(160)), LayerSpec(b, moe), LayerSpec(b, moe, weights_of=1), LayerSpec(a, None)),
                               width=width, vocab=vocab, taps=taps, alpha=alpha, eps=eps, max_pos=4096, name="tiny-zarorax")


def tiny_sikalorn(width=96, vocab=384, eps=1e-5) -> ModelConfig:
    """A small model of the Sikalorn design for tests: every mixer, a layer without feed-forward, three passes over two layers."""
    from .parallel_layers import MixerPairSpec, RecurrentSpec, WindowAttnSpec
    pair = MixerPairSpec(WindowAttnSpec(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.17, rot_dims=16, rope_base=5e4, rope_factor=2.0, window=21),
                         RecurrentSpec("ssd", heads=6, groups=3, dim=20, vdim=16, taps=4, norm_groups=2), 0.8, 0.7)
    delta = RecurrentSpec("delta", heads=4, groups=2, dim=24, vdim=32, taps=4)
    light = RecurrentSpec("lightning", heads=3, groups=3, dim=16, vdim=24, decay=(0.5, 0.9, 0.995))
    specs = [(delta, DenseFFSpec(144)), (pair, DenseFFSpec(120)), (light, None), (pair, DenseFFSpec(64))]
    loop = (1, 3, 3)
    return ModelConfig.layered("Sikalorn", unroll_loop(specs, loop), width=width, vocab=vocab, eps=eps, max_pos=4096, name="tiny-sikalorn", loop=loop)


def tiny_barorax(width=96, vocab=384, eps=1e-5) -> ModelConfig:
    """A small model of the Barorax design for tests: every mixer, a layer without feed-forward, two passes over three layers."""
    from .parallel_layers import SelectiveSpec, WindowAttnSpec
    diff = WindowAttnSpec(heads=4, kv_heads=2, dim=20, vdim=32, scale=0.3, rot_dims=12, rope_base=5e4, kind="attention", row_norm=False,
                          interleaved=True, diff=0.6, gated=True)
    chunk = WindowAttnSpec(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.4, rot_dims=24, rope_base=1e4, kind="attention_2", chunk=21,
                           row_norm=False, interleaved=True, unit=True, sink=True)
    scan = SelectiveSpec(inner=120, state=12, dt_rank=9, taps=4)

    def moe(ff, shared, experts=12, top=3, groups=4, keep=2):
        return RoutedFFSpec(ff, None, experts, top, groups, keep, score="sigmoid", group_best=2, renorm=True, scale=1.7, shared_ff=shared)
    specs = [(scan, moe(40, 56)), (diff, moe(32, 24)), (chunk, None), (scan, moe(24, 48, 8, 2, 1, 1))]
    loop = (1, 4, 2)
    return ModelConfig.layered("Barorax", unroll_loop(specs, loop), width=width, vocab=vocab, eps=eps, max_pos=4096, name="tiny-barorax", loop=loop)


def tiny_derusun(width=96, vocab=384, eps=1e-5, groups=3) -> ModelConfig:
    """A small model of the Derusun design for tests: every mixer, layers without feed-forward, values mixed in two of three layers."""
    from .layered import LatentMixerSpec
    from .parallel_layers import RecurrentSpec, WindowAttnSpec
    latent = LatentMixerSpec("latent_attention", heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=56, rope_base=2e4, scale=0.16, sink=True)
    rec = RecurrentSpec("channel_delta", heads=4, groups=2, dim=24, vdim=32, taps=3, decay_rank=16, gate_rank=8)

    def attn(window, keep, cap, mix=True):
        return WindowAttnSpec(heads=6, kv_heads=2, dim=28, vdim=20, scale=0.2, rot_dims=0, rope_base=1e4, window=window, kind="attention",
                              row_norm=False, bias=True, head_norm=True, softcap=cap, keep_first=keep, head_sink=True, v_mix=mix)
    specs = [(rec, DenseFFSpec(144, 1.5)), (attn(19, 5, 9.0), None), (latent, DenseFFSpec(80, 3.0)), (attn(33, 0, 30.0, False), DenseFFSpec(64, 2.5)),
             (attn(19, 11, 4.0), DenseFFSpec(120, 1.0)), (rec, None)]
    return ModelConfig.layered("Derusun", unroll_loop(specs, None), width=width, vocab=vocab, eps=eps, max_pos=4096, name="tiny-derusun", groups=groups)


@dataclass
class ParallelLayout:
    """Where this rank sits in the TP x PP x EP grid (device coordinates are lexicographic in
    (pp, ep, tp), tp fastest, as in the reference's Placement: crates/skein_cost/src/cluster.rs:100-169)."""
    tp: int = 1
    pp: int = 1
    ep: int = 1
    rank: int = 0

    @property
    def world(self) -> int:
        return self.tp * self.pp * self.ep

    @property
    def tp_rank(self) -> int:
        return self.rank % self.tp

    @property
    def ep_rank(self) -> int:
        return (self.rank // self.tp) % self.ep

    @property
    def pp_rank(self) -> int:
        return self.rank // (self.tp * self.ep)

    def tp_group(self) -> list[int]:
        base = self.rank - self.tp_rank
        return [base + i for i in range(self.tp)]

    def ep_group(self) -> list[int]:
        base = self.pp_rank * self.tp * self.ep + self.tp_rank
        return [base + i * self.tp for i in range(self.ep)]

    def pp_group(self) -> list[int]:
        inner = self.rank % (self.tp * self.ep)
        return [inner + s * self.tp * self.ep for s in range(self.pp)]

    def stage_layers(self, num_layers: int) -> range:
        """Blocks of this pipeline stage; the remainder is spread over the first stages."""
        base, rem = divmod(num_layers, self.pp)
        s = self.pp_rank
        start = s * base + min(s, rem)
        return range(start, start + base + (1 if s < rem else 0))
