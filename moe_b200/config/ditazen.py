"""Typed configuration of the Ditazen design, read from its own config.json keys.

A small decoder whose config.json lists its layers one by one: each entry names its mixer (``type``:
``latent_attention``, attention over one cached latent per position plus a rotated key part, with a sliding
window, a rotation of halves and one output gate a head; ``latent_attention_2``, the same seeing every
earlier position, with the queries through a latent of their own and a rotation of neighbouring pairs
with YaRN scaling; or ``delta``, the gated delta rule), the mixer's sizes (``mixer``) and its feed-forward
(``mlp``: a dense one with the exact GELU, or null for none).  Layers are pre-norm with layer norms that
have a weight and no shift.  A layer with ``weights_of``: j uses layer j's tensors (mixer, feed-forward and
norms) with cache entries and state of its own.  The output projection is the embedding table, its logits
times ``logit_scale``.  Tensors of layer i start with ``l<i>.``.

Every size and every constant that may differ between models comes from config.json; nothing is
derived from one model's values.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .registry import Architecture, ConfigError, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Ditazen"


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


@dataclass(frozen=True)
class RotScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                          # unrotated query/key dimensions of a head
    rot_dim: int                      # rotated ones, whose key all heads share
    vdim: int
    kv_rank: int                      # size of the cached latent
    q_rank: Optional[int]             # size of the queries' latent; None: queries straight from the layer's input
    scale: float                      # factor on the whole score
    window: Optional[int]             # position i sees j with 0 <= i - j < window; None: every earlier one
    rot_base: float
    rot_scaling: Optional[RotScaling]
    neighbours: bool                  # the rotation pairs (2i, 2i + 1) instead of (i, i + rot_dim / 2)


@dataclass(frozen=True)
class DeltaMixerConfig:
    heads: int                        # value heads
    kv_heads: int                     # query/key heads
    dim: int                          # query/key size
    vdim: int                         # value size
    taps: int                         # length of the causal convolutions


@dataclass(frozen=True)
class DitazenLayer:
    type: str
    mixer: Union[LatentMixer, DeltaMixerConfig]
    ff: Optional[int]                 # width of the feed-forward; None: none
    weights_of: Optional[int] = None  # the layer whose tensors it uses


def _latent(m, mw, second: bool) -> LatentMixer:
    rot_dim = _int(m, "rot_dim", mw, low=2)
    if rot_dim % 2:
        _fail(f"{mw}: rot_dim {rot_dim} must be even")
    r, rw = _obj(m, "rot", mw), mw + ".rot"
    if r.get("dims") is not None and _int(r, "dims", rw) != rot_dim:
        _fail(f"{rw}: dims {r['dims']} must be rot_dim {rot_dim}")
    scaling = None
    if r.get("scaling") is not None:
        sc, sw = _obj(r, "scaling", rw), rw + ".scaling"
        scaling = RotScaling(_num(sc, "factor", sw), _num(sc, "original", sw), _num(sc, "fast", sw), _num(sc, "slow", sw))
    window = _int(_obj(m, "mask", mw), "size", mw + ".mask") if m.get("mask") is not None else None
    return LatentMixer(_int(m, "heads", mw), _int(m, "dim", mw), rot_dim, _int(m, "vdim", mw), _int(m, "kv_rank", mw),
                       _int(m, "q_rank", mw) if second else None, _num(m, "scale", mw, positive=False), window,
                       _num(r, "base", rw), scaling, second)


def _delta(m, mw) -> DeltaMixerConfig:
    heads, kv = _int(m, "heads", mw), _int(m, "kv_heads", mw)
    if heads % kv:
        _fail(f"{mw}: heads {heads} is not a multiple of kv_heads {kv}")
    return DeltaMixerConfig(heads, kv, _int(m, "dim", mw), _int(m, "vdim", mw), _int(m, "conv", mw))


_MIXERS = {
    "latent_attention": lambda m, mw: _latent(m, mw, False),
    "latent_attention_2": lambda m, mw: _latent(m, mw, True),
    "delta": _delta,
}


@dataclass(frozen=True)
class DitazenConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[DitazenLayer, ...]
    raw: Tuple[Tuple[str, Any], ...] = ()      # config.json as it was read, for writing it out again

    @staticmethod
    def from_dict(cfg: Dict[str, Any]) -> "DitazenConfig":
        vocab, width = _int(cfg, "vocab", "config.json"), _int(cfg, "width", "config.json")
        eps = _num(_obj(cfg, "norm"), "eps", "norm")
        scale = _num(cfg, "logit_scale", "config.json", positive=False) if cfg.get("logit_scale") is not None else 1.0
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            _fail("'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(e, dict):
                _fail(f"{where} must be an object")
            kind = e.get("type")
            if kind not in _MIXERS:
                _fail(f"{where}: unknown mixer type {kind!r}; known: {', '.join(sorted(_MIXERS))}")
            mixer = _MIXERS[kind](_obj(e, "mixer", where), where + ".mixer")
            ff = None
            if e.get("mlp") is not None:
                ml, mw = _obj(e, "mlp", where), where + ".mlp"
                if ml.get("kind") != "dense":
                    _fail(f"{mw}: unknown kind {ml.get('kind')!r}; known: dense")
                ff = _int(ml, "ff", mw)
            owner = None
            if e.get("weights_of") is not None:
                owner = _int(e, "weights_of", where, low=0)
                if owner >= len(entries) or owner == i:
                    _fail(f"{where}: weights_of {owner} names no other layer of the {len(entries)}")
            layers.append(DitazenLayer(kind, mixer, ff, owner))
        c = DitazenConfig(vocab, width, eps, scale, tuple(layers), tuple(cfg.items()))
        for i, L in enumerate(layers):
            own = layers[c.owner(i)]
            if (L.type, L.mixer, L.ff) != (own.type, own.mixer, own.ff):
                _fail(f"layers[{i}]: differs from layer {c.owner(i)}, whose tensors it uses")
        return c

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses: itself, or the one it names (which may name another)."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if i in seen:
                _fail(f"layers[{i}]: weights_of leads back to itself")
            seen.add(i)
        return i

    def to_dict(self) -> Dict[str, Any]:
        if self.raw:
            return dict(self.raw)

        def mixer(m):
            if isinstance(m, DeltaMixerConfig):
                return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
            d: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                                 "scale": m.scale, "rot": {"dims": m.rot_dim, "base": m.rot_base}}
            if m.q_rank is not None:
                d["q_rank"] = m.q_rank
            if m.window is not None:
                d["mask"] = {"size": m.window}
            if m.rot_scaling is not None:
                s = m.rot_scaling
                d["rot"]["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
            return d

        def layer(l):
            d = {"type": l.type, "mixer": mixer(l.mixer), "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None}
            if l.weights_of is not None:
                d["weights_of"] = l.weights_of
            return d

        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "layers": [layer(l) for l in self.layers]}


def model_spec(c: DitazenConfig) -> ModelSpec:
    """Layer by layer into parts; tensor names are the checkpoint's.  A layer that uses another's tensors is
    that layer run once more with a cache entry of its own."""
    W = c.width

    def norm(name: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("layernorm", {"size": W, "eps": c.norm_eps, "scale": scale, "names": {"weight": ""}}, name)

    def mixer(m, prefix: str) -> PartSpec:
        if isinstance(m, DeltaMixerConfig):
            return PartSpec("delta", {"hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                                      "value_dim": m.vdim, "taps": m.taps, "eps": c.norm_eps}, prefix)
        position: Dict[str, Any] = {"kind": "rotary", "theta": m.rot_base, "rotary_dim": m.rot_dim, "float64": True,
                                    "interleaved": m.neighbours}
        if m.rot_scaling is not None:
            s = m.rot_scaling
            position.update(kind="rotary_yarn", factor=s.factor, original=s.original, fast=s.fast, slow=s.slow)
        return PartSpec(
            "latent_attention",
            {"hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
             "kv_rank": m.kv_rank, "q_rank": m.q_rank, "window": m.window, "scale": m.scale, "eps": c.norm_eps,
             "head_gate": True, "position": position,
             "names": {"q": "q", "q_down": "dq", "q_down_norm": "dq.norm", "q_up": "uq", "down": "dkv",
                       "down_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "gate": "g", "o": "o"}},
            prefix)

    layers, number, ignorable = [], {}, []
    for i, L in enumerate(c.layers):
        if c.owner(i) != i:
            continue
        number[i] = len(layers)
        p = f"l{i}."
        ffn = norm2 = None
        if L.ff is not None:
            norm2 = norm(p + "norm2")
            ffn = PartSpec("dense_mlp", {"hidden_size": W, "size": L.ff, "activation": "gelu",
                                         "names": {"up": "up", "down": "down"}}, p + "mlp.")
        else:
            ignorable += [p + "norm2", p + "norm2.*"]
        layers.append(LayerSpec("prenorm", norm(p + "norm1"), mixer(L.mixer, p + "mix."), norm2, ffn))
    return ModelSpec(
        architecture=ARCHITECTURE,
        hidden_size=W,
        vocab_size=c.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": W, "names": {"weight": ""}}, "embed"),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(number[c.owner(i)], i) for i in range(len(c.layers))),
        # (the factor on the logits rides on the weight of the norm in front of the projection)
        final_norm=norm("final.norm", c.logit_scale),
        head=PartSpec("lm_head", {"vocab_size": c.vocab, "hidden_size": W, "tied": True}, "embed"),
        ignorable=tuple(ignorable),
    )


register_architecture(Architecture(ARCHITECTURE, DitazenConfig.from_dict, model_spec, DitazenConfig.to_dict))
