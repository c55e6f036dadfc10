"""Typed configuration of Pogarax, read from the keys of its config.json.

A Pogarax layer reads the residual stream as it is and norms only what a sublayer gives,
x <- x + m norm1(mixer(x)), x <- x + m norm2(ff(x)), m a constant of the model.  Three mixers:
``channel_delta`` (the gated delta rule behind short convolutions, with a decay per head and key
channel and a gate, both from low-rank products), ``wkv`` (time mixing: every projection reads a
mix of its own of the token's row and the one before, a decay per key channel, a bonus for the
current token) and ``latent_attention`` (queries through a latent, one latent vector and one
rotated key part cached per position, a sliding window, a sink per head; a layer may read another
layer's cache).  Feed-forwards: a dense gated one, or a mixture of gated experts chosen by their
sigmoid scores, whose weight scales the expert's input.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` and ``layers``, a
list of ``{"type", "mixer": {...}, "mlp": {...} | null}``.  Every size and constant that a model
states is read from there; the inner sizes of the low-rank products are read from the stored
tensors.  The design has no position limit.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .hunyuan_dense import ConfigError
from .radorax import Rotary, RotaryScaling

ARCHITECTURE = "Pogarax"
ALIASES = ("pogarax",)
# the design has no limit on positions; the engine's own (``EngineConfig.max_seq_len``) is capped here
MAX_POSITIONS = 1 << 17
# the constant that the design fixes: what is added under the root where q and k become unit vectors
UNIT_KEY_EPS = 1e-6


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None      # only random weights need these two; a stored model's tensors say them
    gate_rank: Optional[int] = None


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int
    decay_rank: Optional[int] = None


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int            # unrotated query/key elements per head
    rot_dim: int        # rotated query/key elements per head (the key's are shared by all heads)
    vdim: int
    kv_rank: int        # width of the cached latent vector
    q_rank: int         # width of the queries' latent
    scale: float
    rot: Rotary
    window: int = 0     # positions that a token sees, its own among them; 0: all
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    expert_ff: int


@dataclass(frozen=True)
class PogaraxLayer:
    type: str
    mixer: Any
    mlp: Any = None


@dataclass(frozen=True)
class PogaraxConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[PogaraxLayer, ...]
    residual_mult: float = 1.0
    eos_token_id: Optional[Tuple[int, ...]] = None

    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "PogaraxConfig":
        def need(obj, key, where):
            if not isinstance(obj, dict) or obj.get(key) is None:
                raise ConfigError(f"config.json lacks '{key}' in {where}")
            return obj[key]

        def optional_int(obj, key):
            return None if obj.get(key) is None else int(obj[key])

        def channel_delta(m, where):
            heads, dim = int(need(m, "heads", where)), int(need(m, "dim", where))
            return ChannelDeltaConfig(heads=heads, kv_heads=int(m.get("kv_heads") or heads), dim=dim,
                                      vdim=int(m.get("vdim") or dim), conv=int(need(m, "conv", where)),
                                      decay_rank=optional_int(m, "decay_rank"), gate_rank=optional_int(m, "gate_rank"))

        def wkv(m, where):
            return WkvConfig(heads=int(need(m, "heads", where)), dim=int(need(m, "dim", where)),
                             decay_rank=optional_int(m, "decay_rank"))

        def latent(m, where):
            rd = need(m, "rot", where)
            sc = rd.get("scaling")
            scaling = None if not sc else RotaryScaling(*(float(need(sc, k, where + ".rot.scaling"))
                                                          for k in ("factor", "original", "fast", "slow")))
            mask = m.get("mask") or {}
            return LatentConfig(
                heads=int(need(m, "heads", where)), dim=int(need(m, "dim", where)),
                rot_dim=int(need(m, "rot_dim", where)), vdim=int(need(m, "vdim", where)),
                kv_rank=int(need(m, "kv_rank", where)), q_rank=int(need(m, "q_rank", where)),
                scale=float(need(m, "scale", where)),
                rot=Rotary(int(need(rd, "dims", where + ".rot")), float(need(rd, "base", where + ".rot")), scaling),
                window=int(mask.get("size") or 0), kv_from=optional_int(m, "kv_from"))

        readers = {"channel_delta": channel_delta, "wkv": wkv, "latent_attention": latent}
        layers: List[PogaraxLayer] = []
        for i, ld in enumerate(need(d, "layers", "the top level")):
            where = f"layers[{i}]"
            kind = str(need(ld, "type", where))
            if kind not in readers:
                raise ConfigError(f"{where}: no mixer '{kind}'; this design has: {', '.join(sorted(readers))}")
            mixer = readers[kind](need(ld, "mixer", where), where + ".mixer")
            md = ld.get("mlp")
            mlp: Any = None
            if md is not None:
                mk = str(need(md, "kind", where + ".mlp"))
                if mk == "dense":
                    mlp = DenseConfig(int(need(md, "ff", where + ".mlp")))
                elif mk == "moe":
                    router = need(md, "router", where + ".mlp")
                    mlp = MoeConfig(experts=int(need(router, "experts", where + ".mlp.router")),
                                    top=int(need(router, "top", where + ".mlp.router")),
                                    expert_ff=int(need(need(md, "expert", where + ".mlp"), "ff", where + ".mlp.expert")))
                else:
                    raise ConfigError(f"{where}.mlp: no feed-forward kind '{mk}'; this design has: dense, moe")
            layers.append(PogaraxLayer(kind, mixer, mlp))
        eos = d.get("eos_token_id")
        eos = (int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos) if eos else None
        mult = d.get("residual_mult")
        cfg = PogaraxConfig(vocab=int(need(d, "vocab", "the top level")), width=int(need(d, "width", "the top level")),
                            eps=float(need(need(d, "norm", "the top level"), "eps", "norm")), layers=tuple(layers),
                            residual_mult=1.0 if mult is None else float(mult), eos_token_id=eos)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be > 0, got {self.eps}")
        for i, layer in enumerate(self.layers):
            m, where = layer.mixer, f"layers[{i}].mixer"
            if isinstance(m, ChannelDeltaConfig):
                if m.heads <= 0 or m.kv_heads <= 0 or m.heads % m.kv_heads or m.dim <= 0 or m.vdim <= 0:
                    raise ConfigError(f"{where}: heads must be a positive multiple of kv_heads, dim and vdim positive")
                if not 1 <= m.conv <= 16:
                    raise ConfigError(f"{where}.conv must be 1 .. 16 taps")
            elif isinstance(m, WkvConfig):
                if m.heads <= 0 or m.dim <= 0:
                    raise ConfigError(f"{where}: heads and dim must be positive")
            else:
                for name in ("heads", "dim", "vdim", "kv_rank", "q_rank"):
                    if getattr(m, name) <= 0:
                        raise ConfigError(f"{where}.{name} must be positive")
                if m.rot_dim < 0 or m.rot_dim % 2 or m.rot.dims % 2 or not 0 <= m.rot.dims <= m.rot_dim:
                    raise ConfigError(f"{where}: rot_dim and rot.dims must be even, 0 <= rot.dims <= rot_dim")
                if not m.rot.base > 0:
                    raise ConfigError(f"{where}.rot.base must be > 0")
                if m.window < 0:
                    raise ConfigError(f"{where}.mask.size must not be negative")
                if m.kv_from is not None:
                    j = m.kv_from
                    o = self.layers[j].mixer if 0 <= j < i else None
                    if not isinstance(o, LatentConfig) or o.kv_from is not None:
                        raise ConfigError(f"{where}.kv_from = {j}: must name an earlier layer that keeps a latent "
                                          "cache of its own")
                    if (o.kv_rank, o.rot_dim, o.rot) != (m.kv_rank, m.rot_dim, m.rot):
                        raise ConfigError(f"layers[{i}] reads the cache of layer {j}: their kv_rank, rot_dim and "
                                          "rot must be equal")
            mlp = layer.mlp
            if isinstance(mlp, DenseConfig) and mlp.ff <= 0:
                raise ConfigError(f"layers[{i}].mlp.ff must be positive")
            if isinstance(mlp, MoeConfig) and not (0 < mlp.top <= mlp.experts and mlp.expert_ff > 0):
                raise ConfigError(f"layers[{i}].mlp: 0 < router.top <= router.experts and expert.ff > 0 are needed")


def _mixer_spec(cfg: PogaraxConfig, i: int, prefix: str):
    from .spec import PartSpec
    m = cfg.layers[i].mixer
    if isinstance(m, ChannelDeltaConfig):
        return PartSpec("mixer", "gated_delta", {
            "hidden_size": cfg.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
            "conv": m.conv, "norm_eps": cfg.eps, "key_eps": UNIT_KEY_EPS, "decay": "channel", "gate": "low_rank",
            "gate_act": "sigmoid", "decay_rank": m.decay_rank, "gate_rank": m.gate_rank}, prefix=prefix)
    if isinstance(m, WkvConfig):
        return PartSpec("mixer", "wkv_time_mix", {
            "hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "norm_eps": cfg.eps,
            "decay_rank": m.decay_rank}, prefix=prefix)
    sc = m.rot.scaling
    position = PartSpec("position", "yarn_rope", {
        "dims": m.rot.dims, "base": m.rot.base, "max_positions": MAX_POSITIONS,
        "scaling": None if sc is None else {"factor": sc.factor, "original": sc.original,
                                            "fast": sc.fast, "slow": sc.slow}})
    # a cache keeps what the widest window among the layers that read it looks back at
    windows = [o.mixer.window for j, o in enumerate(cfg.layers)
               if isinstance(o.mixer, LatentConfig) and (j == i or o.mixer.kv_from == i)]
    return PartSpec("mixer", "latent_attention", {
        "hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
        "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale, "norm_eps": cfg.eps,
        "own_kv": m.kv_from is None, "sink": True, "window": m.window,
        "cache_window": 0 if 0 in windows else max(windows), "position": position,
        "names": {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk",
                  "uv": "uv", "sink": "sink", "out": "o"}}, prefix=prefix)


def _ffn_spec(cfg: PogaraxConfig, mlp, prefix: str):
    from .spec import PartSpec
    if isinstance(mlp, DenseConfig):
        return PartSpec("ffn", "swiglu", {"hidden_size": cfg.width, "intermediate_size": mlp.ff,
                                          "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix=prefix)
    return PartSpec("ffn", "grouped_experts", {
        "hidden_size": cfg.width, "experts": mlp.experts, "top": mlp.top, "expert_size": mlp.expert_ff,
        "scores": "sigmoid", "weight_on": "input"}, prefix=prefix)


def build_spec(cfg: PogaraxConfig):
    """Pogarax as data: per layer a block that norms only the sublayers' results (the residual multiplier is
    those norms' gain), final RMS norm, untied head."""
    from .spec import STREAM_COPY, LayerSpec, ModelSpec, PartSpec, ScheduleStep

    layers, schedule, ignored = [], [], {}
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norm = lambda name: PartSpec("norm", "rms_norm", {"size": cfg.width, "eps": cfg.eps, "weight": name,
                                                          "gain": cfg.residual_mult}, prefix=p)
        parts = {"norm1": norm("norm1"), "mixer": _mixer_spec(cfg, i, p + "mix.")}
        if layer.mlp is not None:
            parts.update(norm2=norm("norm2"), ffn=_ffn_spec(cfg, layer.mlp, p + "mlp."))
        else:
            ignored[p + "norm2"] = "layer has no feed-forward"
        kv_from = getattr(layer.mixer, "kv_from", None)
        if kv_from is not None:
            for name in ("mix.dkv", "mix.dkv.norm"):
                ignored[p + name] = "layer reads another layer's cache"
        layers.append(LayerSpec("output_norm_residual", parts))
        schedule.append(ScheduleStep(i, kv_from))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embed=PartSpec("embed", "token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width,
                                                    "table": "embed", "model_copy": STREAM_COPY}),
        layers=layers, schedule=schedule,
        final_norm=PartSpec("norm", "rms_norm", {"size": cfg.width, "eps": cfg.eps, "weight": "final.norm"}),
        head=PartSpec("head", "lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": None,
                                          "tensor": "head"}),
        eos_token_ids=list(cfg.eos_token_id or ()), ignored_tensors=ignored)
