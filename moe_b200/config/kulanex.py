"""Typed configuration of the Kulanex design, read from its own config.json keys.

A small decoder whose config.json lists its layers one by one: each entry names its mixer (``type``:
"parallel" or "channel_delta"), the mixer's sizes (``mixer``) and its feed-forward (``mlp``: routed experts,
or null for none).  Norms stand on the sublayers' OUTPUT only, RMS norms with a weight stored around zero:
x += m norm1(mixer(x)), x += m norm2(ff(x)), with m = ``residual_mult``; the sublayers read the stream
itself.  The "parallel" mixer runs attention (``left``: a short convolution on q and k, values that are the
convolved keys, one RMS norm over the whole of q and of k, a rotation of pairs (2i, 2i + 1) of part of each head
whose frequencies may be scaled by bands, a given score scale, a sliding window beside which the first positions
stay in sight) beside an exponentially gated matrix memory (``right``) and adds the two outputs with a factor each.
The "channel_delta" mixer is the gated delta rule with a decay a head and key channel.  Experts are picked by
their sigmoid scores, which multiply what the experts read.  Tensors of layer i start with ``l<i>.``.

Every size and every constant that may differ between models comes from config.json (or, for the inner
widths of the delta mixer's narrow projections, from the tensors' shapes); nothing is derived from one model's
values.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .registry import Architecture, ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Kulanex"


def _fail(msg: str):
    raise ConfigError(f"{ARCHITECTURE}: {msg}")


def _obj(cfg, key, where="config.json") -> Dict[str, Any]:
    v = cfg.get(key)
    if not isinstance(v, dict):
        _fail(f"{where} lacks the object '{key}'")
    return v


def _int(cfg, key, where, low=1) -> int:
    v = cfg.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v:
        _fail(f"{where}: '{key}' must be an integer, got {v!r}")
    if int(v) < low:
        _fail(f"{where}: '{key}' must be at least {low}, got {v}")
    return int(v)


def _num(cfg, key, where, positive=True) -> float:
    v = cfg.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        _fail(f"{where}: '{key}' must be a number, got {v!r}")
    if positive and not float(v) > 0:
        _fail(f"{where}: '{key}' must be positive, got {v}")
    return float(v)


def _taps(cfg, where) -> int:
    n = _int(cfg, "conv", where)
    if n > 16:
        _fail(f"{where}: 'conv' must be at most 16, got {n}")
    return n


@dataclass(frozen=True)
class BandScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class LeftAttention:
    heads: int
    kv_heads: int
    dim: int                          # per-head query/key size, and the values' (they are the keys)
    taps: int
    scale: float                      # factor on q . k
    window: Optional[int]             # position i sees j with i - j < window ... (None: every earlier one)
    keep_first: int                   # ... or j < keep_first
    rot_dims: int                     # rotated dimensions of each query/key head (0: none)
    rot_base: float
    scaling: Optional[BandScaling]


@dataclass(frozen=True)
class RightMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelMixer:
    left: LeftAttention
    left_scale: float
    right: RightMemory
    right_scale: float


@dataclass(frozen=True)
class ChannelDelta:
    heads: int                        # value heads
    kv_heads: int                     # query/key heads
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class MoeMlp:
    experts: int
    top: int
    expert_ff: int


@dataclass(frozen=True)
class KulanexLayer:
    type: str
    mixer: Union[ParallelMixer, ChannelDelta]
    mlp: Optional[MoeMlp]


def _heads(m, where) -> Tuple[int, int]:
    heads = _int(m, "heads", where)
    kv = _int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv:
        _fail(f"{where}: heads {heads} is not a multiple of kv_heads {kv}")
    return heads, kv


def _left(l, where) -> LeftAttention:
    heads, kv = _heads(l, where)
    dim = _int(l, "dim", where)
    if l.get("vdim") is not None and _int(l, "vdim", where) != dim:
        _fail(f"{where}: the values are the keys, so vdim {l['vdim']} must equal dim {dim}")
    window, keep = None, 0
    if l.get("mask") is not None:
        m = _obj(l, "mask", where)
        window = _int(m, "size", where + ".mask")
        keep = _int(m, "keep_first", where + ".mask", low=0) if m.get("keep_first") is not None else 0
    dims, base, scaling = 0, 10000.0, None
    if l.get("rot") is not None:
        r, rw = _obj(l, "rot", where), where + ".rot"
        dims, base = _int(r, "dims", rw, low=0), _num(r, "base", rw)
        if dims % 2 or dims > dim:
            _fail(f"{rw}: dims {dims} must be even and at most dim {dim}")
        if r.get("scaling") is not None:
            s, sw = _obj(r, "scaling", rw), rw + ".scaling"
            scaling = BandScaling(*(_num(s, k, sw) for k in ("factor", "low", "high", "original")))
            if scaling.high < scaling.low:
                _fail(f"{sw}: high {scaling.high} is below low {scaling.low}")
    taps = _taps(l, where) if l.get("conv") is not None else 0
    return LeftAttention(heads, kv, dim, taps, _num(l, "scale", where), window, keep, dims, base, scaling)


@dataclass(frozen=True)
class KulanexConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[KulanexLayer, ...]
    raw: Tuple[Tuple[str, Any], ...] = ()      # config.json as it was read, for writing it out again

    @staticmethod
    def from_dict(cfg: Dict[str, Any]) -> "KulanexConfig":
        vocab, width = _int(cfg, "vocab", "config.json"), _int(cfg, "width", "config.json")
        eps = _num(_obj(cfg, "norm"), "eps", "norm")
        mult = _num(cfg, "residual_mult", "config.json", positive=False)
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            _fail("'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(e, dict):
                _fail(f"{where} must be an object")
            kind = e.get("type")
            m, mw = _obj(e, "mixer", where), where + ".mixer"
            if kind == "parallel":
                r, rw = _obj(m, "right", mw), mw + ".right"
                mixer: Union[ParallelMixer, ChannelDelta] = ParallelMixer(
                    _left(_obj(m, "left", mw), mw + ".left"), _num(m, "left_scale", mw, positive=False),
                    RightMemory(_int(r, "heads", rw), _int(r, "dim", rw), _int(r, "vdim", rw), _num(r, "gate_cap", rw)),
                    _num(m, "right_scale", mw, positive=False))
            elif kind == "channel_delta":
                heads, kv = _heads(m, mw)
                mixer = ChannelDelta(heads, kv, _int(m, "dim", mw), _int(m, "vdim", mw), _taps(m, mw))
            else:
                _fail(f"{where}: unknown mixer type {kind!r}; known: parallel, channel_delta")
            mlp = None
            if e.get("mlp") is not None:
                ml, lw = _obj(e, "mlp", where), where + ".mlp"
                if ml.get("kind") != "moe":
                    _fail(f"{lw}: unknown kind {ml.get('kind')!r}; known: moe")
                rt = _obj(ml, "router", lw)
                experts, top = _int(rt, "experts", lw + ".router"), _int(rt, "top", lw + ".router")
                if top > experts:
                    _fail(f"{lw}.router: top {top} exceeds experts {experts}")
                mlp = MoeMlp(experts, top, _int(_obj(ml, "expert", lw), "ff", lw + ".expert"))
            layers.append(KulanexLayer(kind, mixer, mlp))
        return KulanexConfig(vocab, width, eps, mult, tuple(layers), tuple(cfg.items()))

    def to_dict(self) -> Dict[str, Any]:
        if self.raw:
            return dict(self.raw)

        def mixer(m):
            if isinstance(m, ChannelDelta):
                return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
            a, r = m.left, m.right
            left: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale}
            if a.taps:
                left["conv"] = a.taps
            if a.window is not None:
                left["mask"] = {"size": a.window, "keep_first": a.keep_first}
            left["rot"] = {"dims": a.rot_dims, "base": a.rot_base}
            if a.scaling is not None:
                s = a.scaling
                left["rot"]["scaling"] = {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
            return {"left": left, "left_scale": m.left_scale,
                    "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "gate_cap": r.gate_cap},
                    "right_scale": m.right_scale}

        def mlp(f):
            return None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top},
                                           "expert": {"ff": f.expert_ff}}

        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult,
                "layers": [{"type": l.type, "mixer": mixer(l.mixer), "mlp": mlp(l.mlp)} for l in self.layers]}


def model_spec(c: KulanexConfig) -> ModelSpec:
    """Layer by layer into parts; tensor names are the checkpoint's."""
    W = c.width

    def norm(name: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": c.norm_eps, "offset": 1.0, "scale": scale, "names": {"weight": ""}}, name)

    none = PartSpec("none", {"size": W})
    layers = []
    for i, L in enumerate(c.layers):
        p, m = f"l{i}.", L.mixer
        if isinstance(m, ParallelMixer):
            a, r = m.left, m.right
            position: Dict[str, Any] = {"kind": "rotary", "theta": a.rot_base, "rotary_dim": a.rot_dims, "float64": True,
                                        "partial": a.rot_dims < a.dim, "interleaved": True}
            if a.scaling is not None:
                s = a.scaling
                position.update(kind="rotary_bands", factor=s.factor, low=s.low, high=s.high, original=s.original)
            left = {"kind": "gqa_attention", "params": {
                "hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.dim,
                "window": a.window, "keep_first": a.keep_first, "scale": a.scale, "values_are_keys": True,
                "qk_norm": {"eps": c.norm_eps, "whole": True}, "conv": {"taps": a.taps}, "position": position,
                "names": {"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "q_conv": "q.conv",
                          "k_conv": "k.conv"}}}
            right = {"kind": "mlstm", "params": {"hidden_size": W, "num_heads": r.heads, "head_dim": r.dim,
                                                 "value_dim": r.vdim, "gate_cap": r.gate_cap, "eps": c.norm_eps}}
            mixer = PartSpec("side_by_side", {"hidden_size": W, "scales": (m.left_scale, m.right_scale), "left": left,
                                              "right": right}, p + "mix.")
        else:
            mixer = PartSpec("channel_delta", {"hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads,
                                               "head_dim": m.dim, "value_dim": m.vdim, "taps": m.taps, "eps": c.norm_eps},
                             p + "mix.")
        ffn = None
        if L.mlp is not None:
            f = L.mlp
            ffn = PartSpec("routed_experts",
                           {"hidden_size": W, "num_experts": f.experts, "top_k": f.top, "expert_size": f.expert_ff,
                            "score": "sigmoid", "norm_topk_prob": False, "weight_input": True,
                            "names": {"router": "router", "expert_gate": "e{e}.gate", "expert_up": "e{e}.up",
                                      "expert_down": "e{e}.down"}},
                           p + "mlp.")
        layers.append(LayerSpec("sandwich", none, mixer, none if ffn is not None else None, ffn,
                                post1=norm(p + "norm1", c.residual_mult),
                                post2=norm(p + "norm2", c.residual_mult) if ffn is not None else None))
    return ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=W,
        vocab_size=c.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": W, "names": {"weight": "embed"}}, ""),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(l, l, True) for l in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "hidden_size": W, "tied": False, "names": {"weight": ""}}, "head"),
        # a layer without a feed-forward may still carry the norm of one
        ignorable=tuple(f"l{i}.norm2" for i, L in enumerate(c.layers) if L.mlp is None),
    )


register_architecture(Architecture(ARCHITECTURE, KulanexConfig.from_dict, model_spec, KulanexConfig.to_dict))
