"""Typed configuration of Mufalix, read from the keys of its config.json.

A Mufalix layer is x <- x + mixer(norm1(x)), x <- x + ff(norm2(x)).  Two mixers: ``mlstm`` (a matrix memory
per head with exponential gates under a running maximum) and ``parallel``, two mixers side by side on the same
input: grouped-query attention (biases, a norm per query and key head before a partial rotation, a sliding
window, a learnt sink per head, an output gate) and a gated linear recurrence behind a short convolution;
half the sum of their results, each normed over the width.  Feed-forwards are experts of a squared relu,
chosen by sigmoid scores plus a correction and weighted by the chosen scores over their sum.  A range of layers
may run several times in a row with the same weights, each pass with caches and states of its own; a pass
begins with a product of the stream beside the embedding output.

config.json: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``loop`` ({start, stop,
times}, optional) and ``layers``, a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``.  Every size and
constant that a model states is read from there.  The design has no position limit.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .hunyuan_dense import ConfigError
from .vodelix import ATTENTION_HEAD_SIZES, Loop

ARCHITECTURE = "Mufalix"
ALIASES = ("mufalix",)
# the design has no limit on positions; the engine's own (``EngineConfig.max_seq_len``) is capped here
MAX_POSITIONS = 1 << 17
# the constant that the design fixes: what is added to the matrix memory's normaliser
DEN_EPS = 1e-6
# widest head that any attention kernel takes
MAX_HEAD = 512


@dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                  # positions that a token sees, its own among them; 0: all
    rot_dims: int = 0
    rot_base: float = 10000.0
    scaling: Optional[WavelengthScaling] = None


@dataclass(frozen=True)
class RecurrenceConfig:
    width: int                       # channels
    blocks: int
    conv: int


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: RecurrenceConfig


@dataclass(frozen=True)
class MlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    scale: float
    expert_ff: int


@dataclass(frozen=True)
class MufalixLayer:
    type: str
    mixer: Any
    mlp: Optional[MoeConfig] = None


@dataclass(frozen=True)
class MufalixConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[MufalixLayer, ...]
    embedding_scale: float = 1.0
    loop: Optional[Loop] = None
    eos_token_id: Optional[Tuple[int, ...]] = None

    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "MufalixConfig":
        def need(obj, key, where):
            if not isinstance(obj, dict) or obj.get(key) is None:
                raise ConfigError(f"config.json lacks '{key}' in {where}")
            return obj[key]

        def attention(m, where):
            heads, dim = int(need(m, "heads", where)), int(need(m, "dim", where))
            rot = m.get("rot") or {}
            sc = rot.get("scaling")
            scaling = None if not sc else WavelengthScaling(*(float(need(sc, k, where + ".rot.scaling"))
                                                              for k in ("factor", "low", "high", "original")))
            return AttentionConfig(
                heads=heads, kv_heads=int(m.get("kv_heads") or heads), dim=dim, vdim=int(m.get("vdim") or dim),
                scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5,
                window=int((m.get("mask") or {}).get("size") or 0), rot_dims=int(rot.get("dims") or 0),
                rot_base=float(rot.get("base") or 10000.0), scaling=scaling)

        layers: List[MufalixLayer] = []
        for i, ld in enumerate(need(d, "layers", "the top level")):
            where = f"layers[{i}]"
            kind, m = str(need(ld, "type", where)), need(ld, "mixer", where)
            where += ".mixer"
            if kind == "parallel":
                rt = need(m, "right", where)
                mixer: Any = ParallelConfig(
                    attention(need(m, "left", where), where + ".left"),
                    RecurrenceConfig(*(int(need(rt, k, where + ".right")) for k in ("width", "blocks", "conv"))))
            elif kind == "mlstm":
                dim = int(need(m, "dim", where))
                mixer = MlstmConfig(heads=int(need(m, "heads", where)), dim=dim, vdim=int(m.get("vdim") or dim),
                                    gate_cap=float(need(m, "gate_cap", where)))
            else:
                raise ConfigError(f"layers[{i}]: no mixer '{kind}'; this design has: mlstm, parallel")
            md, mlp = ld.get("mlp"), None
            if md is not None:
                where = f"layers[{i}].mlp"
                if str(md.get("kind") or "moe") != "moe":
                    raise ConfigError(f"{where}: no feed-forward kind '{md['kind']}'; this design has: moe")
                router = need(md, "router", where)
                scale = router.get("scale")
                mlp = MoeConfig(experts=int(need(router, "experts", where + ".router")),
                                top=int(need(router, "top", where + ".router")), scale=1.0 if scale is None else float(scale),
                                expert_ff=int(need(need(md, "expert", where), "ff", where + ".expert")))
            layers.append(MufalixLayer(kind, mixer, mlp))
        lp = d.get("loop")
        loop = None if not lp else Loop(*(int(need(lp, k, "loop")) for k in ("start", "stop", "times")))
        scale = (d.get("embedding") or {}).get("scale")
        eos = d.get("eos_token_id")
        eos = (int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos) if eos else None
        cfg = MufalixConfig(vocab=int(need(d, "vocab", "the top level")), width=int(need(d, "width", "the top level")),
                            eps=float(need(need(d, "norm", "the top level"), "eps", "norm")), layers=tuple(layers),
                            embedding_scale=1.0 if scale is None else float(scale), loop=loop, eos_token_id=eos)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be > 0, got {self.eps}")
        for i, layer in enumerate(self.layers):
            m, where = layer.mixer, f"layers[{i}].mixer"
            if isinstance(m, ParallelConfig):
                lt, rt = m.left, m.right
                if lt.heads <= 0 or lt.kv_heads <= 0 or lt.heads % lt.kv_heads or not 0 < lt.dim <= MAX_HEAD \
                        or not 0 < lt.vdim <= MAX_HEAD:
                    raise ConfigError(f"{where}.left: heads must be a positive multiple of kv_heads, dim and vdim "
                                      f"1 .. {MAX_HEAD}")
                if lt.rot_dims < 0 or lt.rot_dims % 2 or lt.rot_dims > lt.dim or not lt.rot_base > 0:
                    raise ConfigError(f"{where}.left.rot: dims must be even and at most dim, base positive")
                if lt.window < 0:
                    raise ConfigError(f"{where}.left.mask.size must not be negative")
                if rt.blocks <= 0 or rt.width <= 0 or rt.width % rt.blocks or not 1 <= rt.conv <= 16:
                    raise ConfigError(f"{where}.right: width must be a positive multiple of blocks, conv 1 .. 16 taps")
            elif m.heads <= 0 or m.dim <= 0 or m.vdim <= 0 or not m.gate_cap > 0:
                raise ConfigError(f"{where}: heads, dim, vdim and gate_cap must be positive")
            mlp = layer.mlp
            if mlp is not None and not (0 < mlp.top <= mlp.experts and mlp.expert_ff > 0):
                raise ConfigError(f"layers[{i}].mlp: 0 < router.top <= router.experts and expert.ff > 0 are needed")
        lp = self.loop
        if lp is not None and (not 0 <= lp.start < lp.stop <= len(self.layers) or lp.times < 1):
            raise ConfigError("loop: 0 <= start < stop <= number of layers and times >= 1 are needed")

    def runs(self) -> List[Tuple[int, bool]]:
        """The layers in the order they run: (layer, whether a pass begins with this run)."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, False) for i in range(n)]
        one_pass = [(i, i == lp.start) for i in range(lp.start, lp.stop)]
        return [(i, False) for i in range(lp.start)] + one_pass * lp.times + [(i, False) for i in range(lp.stop, n)]


def stored_head_size(dim: int, vdim: int) -> int:
    """The head size that keys and values are stored at: the smallest one that the attention kernels are compiled for,
    or, for wider heads, the even number above both (the FP32-core kernel takes those)."""
    fit = [s for s in ATTENTION_HEAD_SIZES if s >= max(dim, vdim)]
    return fit[0] if fit else -(-max(dim, vdim) // 2) * 2


def _parallel_spec(cfg: MufalixConfig, m: ParallelConfig, prefix: str):
    from .spec import PartSpec
    lt, rt, sc = m.left, m.right, m.left.scaling
    position = None
    if lt.rot_dims:
        position = PartSpec("position", "wavelength_rope", {
            "dims": lt.rot_dims, "base": lt.rot_base, "max_positions": MAX_POSITIONS,
            "scaling": None if sc is None else {"factor": sc.factor, "low": sc.low, "high": sc.high,
                                                "original": sc.original}})
    head = stored_head_size(lt.dim, lt.vdim)
    left = PartSpec("mixer", "gqa_attention", {
        "hidden_size": cfg.width, "num_heads": lt.heads, "num_kv_heads": lt.kv_heads, "head_dim": head,
        "key_dim": lt.dim, "value_dim": lt.vdim, "bias": True, "qk_norm": True, "qk_norm_eps": cfg.eps,
        "qk_norm_order": "before_rope", "rotary_dim": lt.rot_dims or None, "position": position, "window": lt.window,
        "scale": lt.scale, "sink": True, "gate": True,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b",
                  "o_bias": "o.b", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "sink": "sink"}},
                    prefix=prefix + "left.")
    right = PartSpec("mixer", "gated_linear_recurrence", {
        "hidden_size": cfg.width, "channels": rt.width, "blocks": rt.blocks, "conv": rt.conv}, prefix=prefix + "right.")
    return PartSpec("mixer", "parallel_pair", {
        "hidden_size": cfg.width, "eps": cfg.eps, "left": left, "right": right,
        "left_norm": "left.out", "right_norm": "right.out", "head_dim": head}, prefix=prefix)


def _mlstm_spec(cfg: MufalixConfig, m: MlstmConfig, prefix: str):
    from .spec import PartSpec
    return PartSpec("mixer", "exponential_gates", {
        "hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap,
        "norm_eps": cfg.eps, "den_eps": DEN_EPS}, prefix=prefix)


def build_spec(cfg: MufalixConfig):
    """Mufalix as data: per layer a pre-norm block; the schedule names the looped layers once per pass, and the first
    layer of every pass has an entry."""
    from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleStep

    layers, ignored = [], {}
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norm = lambda name: PartSpec("norm", "rms_norm", {"size": cfg.width, "eps": cfg.eps, "weight": name}, prefix=p)
        mixer = (_parallel_spec if layer.type == "parallel" else _mlstm_spec)(cfg, layer.mixer, p + "mix.")
        parts = {"norm1": norm("norm1"), "mixer": mixer}
        if layer.mlp is not None:
            parts.update(norm2=norm("norm2"), ffn=PartSpec("ffn", "routed_experts", {
                "hidden_size": cfg.width, "experts": layer.mlp.experts, "top": layer.mlp.top,
                "expert_size": layer.mlp.expert_ff, "act": "relu2", "scores": "sigmoid", "correction": "correction",
                "route_scale": layer.mlp.scale}, prefix=p + "mlp."))
        else:
            ignored[p + "norm2"] = "layer has no feed-forward"
        layers.append(LayerSpec("prenorm_residual", parts))
    if cfg.loop is None:
        ignored["loop.in"] = "no layer is repeated"
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embed=PartSpec("embed", "token_embedding", {
            "vocab_size": cfg.vocab, "hidden_size": cfg.width, "table": "embed", "scale": cfg.embedding_scale,
            "keep_copy": cfg.loop is not None}),
        layers=layers, schedule=[ScheduleStep(i, None, {} if enters else None) for i, enters in cfg.runs()],
        final_norm=PartSpec("norm", "rms_norm", {"size": cfg.width, "eps": cfg.eps, "weight": "final.norm"}),
        head=PartSpec("head", "lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": None,
                                          "tensor": "head"}),
        entry=None if cfg.loop is None else PartSpec("entry", "pass_projection", {"size": cfg.width, "tensor": "loop.in"}),
        eos_token_ids=list(cfg.eos_token_id or ()), ignored_tensors=ignored)
