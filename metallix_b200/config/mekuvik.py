"""Typed configuration of the Mekuvik decoder, read from ``config.json``.

A Mekuvik model is a stack of layers over one float32 residual stream that
starts as ``embed[token]`` =: x0. A layer has one norm, whose output both of its
sublayers read:

    h = norm1(x);   x <- x + (mixer(h) + ff(h))

with RMS norms times a plain weight; a layer may have no feed-forward. With
``loop``, the layers start .. stop - 1 run ``times`` times in a row with the same
weights, each pass with a cache or state of its own; right before every pass but
the first x <- x + x0. The logits are embed x final_norm(x) * ``logit_scale``. The
mixer is one of

* ``lightning``: linear attention with a constant decay per head. q = silu(Wq h),
  k = silu(Wk h) (``heads`` of ``dim``), v = silu(Wv h) (``heads`` of ``vdim``); per
  head S <- decay S + k v^T, o = S^T q; the heads side by side over their common
  root mean square, times a weight, times sigmoid(Wg h), then Wo. S is state of a
  request;
* ``attention``: grouped-query attention; RMS norms over all of a token's queries
  and over all of its keys, ahead of the rotation of neighbouring pairs among a
  head's first ``rot.dims`` values; the score scale is the configuration's; a query
  sees the last ``mask.size`` positions and the first ``mask.keep_first`` ones;
* ``latent_attention``: queries through a latent of ``q_rank`` values with a norm,
  per head [``dim`` unrotated | ``rot_dim`` rotated]; a down-projection gives
  ``kv_rank`` values that are normed (the latent) and ``rot_dim`` values that are
  rotated (one key part for all heads); per head the unrotated key and the value
  are up-projections of the latent; rotation of neighbouring pairs
  (``rot.scaling``, optional: factor, original, fast, slow); causal; the heads side
  by side times sigmoid(Wg h), then Wo.

The feed-forward is ``dense``, Wdown (silu(Wgate h) * (Wup h)); or ``moe``:
``router.experts`` experts Wdown gelu(Wup h) (gelu in its exact form) of which a
token uses the ``router.top`` with the largest sigmoid scores of the router's
float32 logits; a chosen expert reads its score times h, and what the chosen leave
is added up; a shared expert of the same form (``shared.ff``, optional) reads h and
is added.

``config.json``::

    {"architecture": "Mekuvik", "vocab": V, "width": W, "norm": {"eps": e}, "logit_scale": c,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "lightning", "mixer": {"heads": H, "dim": D, "vdim": Dv, "decay": [H numbers]},
                 "mlp": {"kind": "dense", "ff": F}},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": c,
                           "rot": {"base": b, "dims": R}, "mask": {"size": w, "keep_first": k}},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": Fs}, "router": {"experts": E, "top": k}}},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": D, "rot_dim": R, "vdim": Dv, "q_rank": rq, "kv_rank": r, "scale": c,
                           "rot": {"base": b, "dims": R, "scaling": {"factor": f, "original": n, "fast": x, "slow": y}}},
                 "mlp": null}]}

Tensors (linear weights ``[out, in]``): ``embed`` [V, W], ``final.norm`` [W]; per
layer i ``l<i>.norm1`` [W]; under ``l<i>.mix`` a lightning has ``q``, ``k`` [H D, W],
``v``, ``g`` [H Dv, W], ``norm`` [H Dv], ``o`` [W, H Dv]; an attention has ``q`` [H D, W],
``k`` [G D, W], ``v`` [G Dv, W], ``q.norm`` [H D], ``k.norm`` [G D], ``o`` [W, H Dv]; a
latent_attention has ``dq`` [rq, W], ``dq.norm`` [rq], ``uq`` [H (D + R), rq], ``dkv``
[r + R, W], ``dkv.norm`` [r], ``uk`` [H D, r], ``uv`` [H Dv, r], ``g`` [H Dv, W], ``o``
[W, H Dv]. Under ``l<i>.mlp`` a dense feed-forward has ``gate``, ``up`` [F, W], ``down``
[W, F]; a moe has ``e<j>.up`` [F, W], ``e<j>.down`` [W, F], ``router`` [E, W] and, with
a shared expert, ``shared.up`` [Fs, W], ``shared.down`` [W, Fs].
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .dimorax import GatedDense, Rotation
from .mekazen import MAX_POSITIONS, _count, _number, _object
from .qwen3 import ConfigError
from .sadosun import _positive
from .spec import LayerRun, LayerSpec, ModelSpec, PartSpec


def _optional_count(raw: Mapping[str, Any], key: str, where: str, default: int) -> int:
    return _count(raw, key, where) if raw.get(key) is not None else default


def _paired(rot: Optional[Rotation], head_dim: int) -> Optional[PartSpec]:
    """The rotation of neighbouring pairs with a rotation's parameters."""
    return PartSpec("rope_interleaved", dict(rot.part(head_dim).params)) if rot is not None else None


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "LightningMixer":
        raw = _object(raw, where)
        heads, dim, given = _count(raw, "heads", where), _count(raw, "dim", where), raw.get("decay")
        if not isinstance(given, list) or len(given) != heads:
            raise ConfigError("InvalidDecay", f"{where}.decay must be a list of {heads} numbers, one per head")
        decay = tuple(_number({"decay": value}, "decay", where) for value in given)
        if not all(0.0 <= value <= 1.0 for value in decay):
            raise ConfigError("InvalidDecay", f"{where}.decay must lie in [0, 1], got {given}")
        return cls(heads=heads, dim=dim, vdim=_optional_count(raw, "vdim", where, dim), decay=decay)

    def to_dict(self) -> Dict[str, Any]:
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        qk, v = self.heads * self.dim, self.heads * self.vdim
        return {f"{base}.q": (qk, w), f"{base}.k": (qk, w), f"{base}.v": (v, w), f"{base}.g": (v, w), f"{base}.o": (w, v),
                f"{base}.norm": (v,)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        return PartSpec("lightning", {
            "hidden_size": w, "num_heads": self.heads, "head_dim": self.dim, "value_dim": self.vdim, "decay": self.decay,
            "eps": eps, "q_proj": f"{base}.q", "k_proj": f"{base}.k", "v_proj": f"{base}.v", "gate_proj": f"{base}.g",
            "norm": f"{base}.norm", "o_proj": f"{base}.o"})


@dataclass(frozen=True)
class KeptWindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                     # 0: every earlier position is seen
    keep_first: int                 # the first positions that stay visible beside the window
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "KeptWindowAttention":
        raw = _object(raw, where)
        heads, dim = _count(raw, "heads", where), _count(raw, "dim", where)
        kv_heads = _optional_count(raw, "kv_heads", where, heads)
        if heads % kv_heads:
            raise ConfigError("InvalidGroupedQueryLayout", f"{where}: {heads} query heads over {kv_heads} key/value heads")
        if dim % 2:
            raise ConfigError("OddHeadDimension", f"{where}.dim {dim}")
        window = keep = 0
        if raw.get("mask") is not None:
            mask = _object(raw["mask"], f"{where}.mask")
            window, keep = _count(mask, "size", f"{where}.mask"), mask.get("keep_first") or 0
            if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
                raise ConfigError("Json", f"{where}.mask.keep_first must be a number of positions, got {keep!r}")
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_optional_count(raw, "vdim", where, dim),
                   scale=_positive(raw, "scale", where), window=window, keep_first=keep,
                   rot=Rotation.from_dict(raw["rot"], f"{where}.rot", dim) if raw.get("rot") is not None else None)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads}
        if self.window:
            out["mask"] = {"keep_first": self.keep_first, "size": self.window}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        out.update(scale=self.scale, vdim=self.vdim)
        return out

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        q, k = self.heads * self.dim, self.kv_heads * self.dim
        return {f"{base}.q": (q, w), f"{base}.k": (k, w), f"{base}.v": (self.kv_heads * self.vdim, w),
                f"{base}.q.norm": (q,), f"{base}.k.norm": (k,), f"{base}.o": (w, self.heads * self.vdim)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        norm = lambda name, heads: PartSpec("rmsnorm", {"size": heads * self.dim, "eps": eps, "weight": name})
        return PartSpec("gqa_attention", {
            "hidden_size": w, "num_heads": self.heads, "num_kv_heads": self.kv_heads, "head_dim": self.dim,
            "value_dim": self.vdim, "scale": self.scale, "softcap": None, "window": self.window or None, "chunk": None,
            "keep_first": self.keep_first, "q_proj": f"{base}.q", "k_proj": f"{base}.k", "v_proj": f"{base}.v",
            "gate_proj": None, "o_proj": f"{base}.o", "qk_norm_scope": "projection",
            "q_norm": norm(f"{base}.q.norm", self.heads), "k_norm": norm(f"{base}.k.norm", self.kv_heads),
            "position": _paired(self.rot, self.dim), "value_position": None, "sink": None, "pad_heads": True})


@dataclass(frozen=True)
class GatedLatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "GatedLatentAttention":
        raw = _object(raw, where)
        rot_dim, dim = _count(raw, "rot_dim", where), _count(raw, "dim", where)
        rot = Rotation.from_dict(raw["rot"], f"{where}.rot", rot_dim) if raw.get("rot") is not None else None
        if rot is not None and rot.dims != rot_dim:
            raise ConfigError("InvalidRotaryWidth", f"{where}: rot.dims {rot.dims} must be rot_dim {rot_dim}")
        return cls(heads=_count(raw, "heads", where), dim=dim, rot_dim=rot_dim,
                   vdim=_optional_count(raw, "vdim", where, dim), q_rank=_count(raw, "q_rank", where),
                   kv_rank=_count(raw, "kv_rank", where), scale=_positive(raw, "scale", where), rot=rot)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        out.update(rot_dim=self.rot_dim, scale=self.scale, vdim=self.vdim)
        return out

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        H, r = self.heads, self.kv_rank
        return {f"{base}.dq": (self.q_rank, w), f"{base}.dq.norm": (self.q_rank,),
                f"{base}.uq": (H * (self.dim + self.rot_dim), self.q_rank), f"{base}.dkv": (r + self.rot_dim, w),
                f"{base}.dkv.norm": (r,), f"{base}.uk": (H * self.dim, r), f"{base}.uv": (H * self.vdim, r),
                f"{base}.g": (H * self.vdim, w), f"{base}.o": (w, H * self.vdim)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        return PartSpec("latent_attention", {
            "hidden_size": w, "num_heads": self.heads, "head_dim": self.dim, "rotary_head_dim": self.rot_dim,
            "value_dim": self.vdim, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale, "eps": eps,
            "q_down_proj": f"{base}.dq", "q_up_proj": f"{base}.uq", "kv_down_proj": f"{base}.dkv",
            "k_up_proj": f"{base}.uk", "v_up_proj": f"{base}.uv", "gate_proj": f"{base}.g", "o_proj": f"{base}.o",
            "q_norm": PartSpec("rmsnorm", {"size": self.q_rank, "eps": eps, "weight": f"{base}.dq.norm"}),
            "kv_norm": PartSpec("rmsnorm", {"size": self.kv_rank, "eps": eps, "weight": f"{base}.dkv.norm"}),
            "position": _paired(self.rot, self.rot_dim), "window": None, "sink": None, "cache_mode": "auto"})


_MIXERS = {"lightning": LightningMixer, "attention": KeptWindowAttention, "latent_attention": GatedLatentAttention}


@dataclass(frozen=True)
class WeighedExperts:
    ff: int
    experts: int
    top: int
    shared_ff: int          # 0: no expert that every token uses

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "WeighedExperts":
        router = _object(raw.get("router"), f"{where}.router")
        experts, top = _count(router, "experts", f"{where}.router"), _count(router, "top", f"{where}.router")
        if top > experts:
            raise ConfigError("Json", f"{where}.router: top {top} of {experts} experts")
        shared = 0
        if raw.get("shared") is not None:
            shared = _count(_object(raw["shared"], f"{where}.shared"), "ff", f"{where}.shared")
        return cls(ff=_count(_object(raw.get("expert"), f"{where}.expert"), "ff", f"{where}.expert"), experts=experts,
                   top=top, shared_ff=shared)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        shapes: Dict[str, tuple] = {}
        for index in range(self.experts):
            shapes.update({f"{base}.e{index}.up": (self.ff, w), f"{base}.e{index}.down": (w, self.ff)})
        shapes[f"{base}.router"] = (self.experts, w)
        if self.shared_ff:
            shapes.update({f"{base}.shared.up": (self.shared_ff, w), f"{base}.shared.down": (w, self.shared_ff)})
        return shapes

    def part(self, base: str, w: int) -> PartSpec:
        shared = PartSpec("dense_ff", {"hidden_size": w, "intermediate_size": self.shared_ff, "activation": "gelu",
                                       "up_proj": f"{base}.shared.up", "down_proj": f"{base}.shared.down"})
        return PartSpec("routed_experts", {
            "hidden_size": w, "intermediate_size": self.ff, "experts": self.experts, "identity": 0, "top": self.top,
            "activation": "gelu", "scores": "sigmoid", "normalized": False, "weigh_input": True,
            "up_proj": base + ".e{}.up", "down_proj": base + ".e{}.down", "router": f"{base}.router",
            "shared": shared if self.shared_ff else None})


def _feed_forward(raw: Mapping[str, Any], where: str):
    raw = _object(raw, where)
    kind = raw.get("kind")
    if kind == "dense":
        return GatedDense(ff=_count(raw, "ff", where))
    if kind == "moe":
        return WeighedExperts.from_dict(raw, where)
    raise ConfigError("UnsupportedFeedForward", f"{where}.kind {kind!r}; 'dense' or 'moe'")


@dataclass(frozen=True)
class MekuvikLayer:
    kind: str
    mixer: object
    mlp: Optional[object]       # None: no feed-forward

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "MekuvikLayer":
        raw = _object(raw, where)
        kind = raw.get("type")
        if kind not in _MIXERS:
            raise ConfigError("UnsupportedLayerType", f"{where}.type {kind!r}; this design has {sorted(_MIXERS)}")
        mlp = _feed_forward(raw["mlp"], f"{where}.mlp") if raw.get("mlp") is not None else None
        return cls(kind=kind, mixer=_MIXERS[kind].from_dict(raw.get("mixer"), f"{where}.mixer"), mlp=mlp)

    def to_dict(self) -> Dict[str, Any]:
        return {"mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None,
                "type": self.kind}

    def feed_forward_part(self, base: str, w: int) -> Optional[PartSpec]:
        if self.mlp is None:
            return None
        return self.mlp.part(base, w, "silu") if isinstance(self.mlp, GatedDense) else self.mlp.part(base, w)


@dataclass(frozen=True)
class MekuvikConfig:
    """Sizes and constants of one Mekuvik checkpoint."""

    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[MekuvikLayer, ...]
    logit_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    eos_token_ids: tuple = ()

    ARCHITECTURE = "Mekuvik"
    MODEL_TYPE = "mekuvik"

    @classmethod
    def parse(cls, text: str) -> "MekuvikConfig":
        try:
            raw = json.loads(text)
        except json.JSONDecodeError as error:
            raise ConfigError("Json", str(error)) from None
        return cls.from_dict(_object(raw, "config.json"))

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "MekuvikConfig":
        if raw.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError("UnsupportedModelType", f"architecture {raw.get('architecture')!r}")
        vocab, width = _count(raw, "vocab", "config"), _count(raw, "width", "config")
        if width % 8:
            raise ConfigError("MissingDimension", f"width {width} must be a multiple of 8")
        eps = _number(_object(raw.get("norm"), "norm"), "eps", "norm")
        if eps <= 0.0:
            raise ConfigError("InvalidRmsNormEpsilon", str(eps))
        given = raw.get("layers")
        if not isinstance(given, list) or not given:
            raise ConfigError("MissingDimension", "layers must be a list of at least one layer")
        layers = tuple(MekuvikLayer.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(given))
        loop = None
        if raw.get("loop") is not None:
            loop = _object(raw["loop"], "loop")
            start = loop.get("start")
            if isinstance(start, bool) or not isinstance(start, int) or start < 0:
                raise ConfigError("Json", f"loop.start must be a layer's index, got {start!r}")
            stop, times = _count(loop, "stop", "loop"), _count(loop, "times", "loop")
            if not start < stop <= len(layers):
                raise ConfigError("Json", f"loop: layers {start} .. {stop - 1} of {len(layers)}")
            loop = (start, stop, times)
        scale = _number(raw, "logit_scale", "config") if raw.get("logit_scale") is not None else 1.0
        return cls(vocab=vocab, width=width, norm_eps=eps, layers=layers, logit_scale=scale, loop=loop)

    # ------------------------------------------------------------ derived facts
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    def parameter_count(self) -> int:
        return sum(math.prod(shape) for shape in self.tensor_shapes().values())

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.ARCHITECTURE, "layers": [layer.to_dict() for layer in self.layers],
               "logit_scale": self.logit_scale}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        out.update({"norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width})
        return out

    # ------------------------------------------------------------- model spec
    def _order(self) -> Tuple[LayerRun, ...]:
        """Layers in the order they run; every pass after the first has cache entries behind all layers' own and meets
        the embedding output ahead of its first layer."""
        count = len(self.layers)
        if self.loop is None:
            return tuple(LayerRun(layer=index) for index in range(count))
        start, stop, times = self.loop
        runs = [LayerRun(layer=index) for index in range(stop)]
        for turn in range(1, times):
            for index in range(start, stop):
                entry = count + (turn - 1) * (stop - start) + index - start
                runs.append(LayerRun(layer=index, cache=entry, join=0 if index == start else None, turn=turn))
        return tuple(runs + [LayerRun(layer=index) for index in range(stop, count)])

    def to_model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps
        norm = lambda name, scale=1.0: PartSpec("rmsnorm", {"size": w, "eps": eps, "weight": name, "scale": scale})
        layers = []
        for index, layer in enumerate(self.layers):
            base = f"l{index}"
            layers.append(LayerSpec(
                name=base, block=PartSpec("parallel_residual", {"hidden_size": w, "residual_scale": 1.0, "shared_norm": True}),
                mixer=layer.mixer.part(f"{base}.mix", w, eps), feed_forward=layer.feed_forward_part(f"{base}.mlp", w),
                mixer_norm=norm(f"{base}.norm1"), feed_forward_norm=None))
        order = self._order()
        spec = ModelSpec(
            architecture=self.ARCHITECTURE, hidden_size=w, vocab_size=self.vocab, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": w, "weight": "embed"}),
            # the logits' constant rides in the last norm's weight
            layers=tuple(layers), order=order, final_norm=norm("final.norm", self.logit_scale),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": w, "weight": "embed", "softcap": None}),
            joins=(PartSpec("add_first", {"hidden_size": w}),) if any(run.join is not None for run in order) else ())
        spec.validate()
        return spec

    # ------------------------------------------------ tensors of a checkpoint
    def tensor_shapes(self) -> Dict[str, tuple]:
        w = self.width
        shapes: Dict[str, tuple] = {"embed": (self.vocab, w)}
        for index, layer in enumerate(self.layers):
            base = f"l{index}"
            shapes[f"{base}.norm1"] = (w,)
            shapes.update(layer.mixer.shapes(f"{base}.mix", w))
            if layer.mlp is not None:
                shapes.update(layer.mlp.shapes(f"{base}.mlp", w))
        shapes["final.norm"] = (w,)
        return shapes

    def ignored_tensors(self) -> tuple:
        return ()

    def norm_tensor(self, name: str):
        """How a tensor of random weights is drawn: False for a matrix
        (N(0, 0.02)); "one" for a factor near 1."""
        return "one" if name.rsplit(".", 1)[-1] in ("norm1", "norm") else False
