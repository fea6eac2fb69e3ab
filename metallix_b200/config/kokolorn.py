"""Typed configuration of the Kokolorn decoder, read from ``config.json``.

A Kokolorn model is a stack of pre-norm layers over one float32 residual stream
that starts as ``embed[token] * embedding.scale``,

    x <- x + mixer(norm1(x));   x <- x + ff(norm2(x))

with RMS norms whose stored weight lies around zero (the factor is 1 + w); a
layer may have no feed-forward. With ``loop``, the layers start .. stop - 1 run
``times`` times in a row with the same weights, each pass with a cache or state
of its own; right before a pass x <- W_in [x; x0], x0 being the stream as the
embedding left it, and the pass's vector is added. The logits are
embed x final_norm(x) (the table without its scale). The mixer is one of

* ``attention``: grouped-query attention whose values are the keys as projected
  (bias included, ahead of the key norm); q and k have biases and RMS norms per
  head; no rotation, but q is multiplied by 1 + coef ln(floor((p + 1) / every) +
  1) at position p (``q_temp``, optional); the score scale is the
  configuration's; the mask is causal;
* ``delta``: the gated delta rule with one decay per head. q and k
  (``kv_heads`` groups of ``dim``) and v (``heads`` of ``vdim``) pass a short
  causal convolution over time and silu; unit norms, write strength, decay,
  S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; each head's o over
  its root mean square, times a weight over vdim, times silu(Wg h), then Wo;
* ``parallel``: two mixers on the same input, half the sum of their outputs,
  each over its own root mean square times a weight over the width. ``left`` is
  the attention without the head norms, with a bias on its output projection
  and a learned bias per head and distance on its scores (a table whose rows
  are distances, logarithmic beyond its first half, up to ``bias_max``); ``right``
  is the state-space dual (Mamba-2) with ``groups`` of B and C, a gate ahead of
  its norm and the norm in ``norm_groups`` parts.

The feed-forward is ``dense``, with g = min(Wgate h, limit) and u = clamp(Wup h,
-limit, limit): Wdown (g sigmoid(1.702 g) (u + 1)); or ``moe``:
``router.experts`` experts Wdown max(Wup h, 0)^2 of which a token uses the
``router.top`` with the largest router logits (bias included), weighted by the
softmax over the chosen logits, and a shared expert of the same form
(``shared.ff``, optional) added for every token.

``config.json``::

    {"architecture": "Kokolorn", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": c,
                           "q_temp": {"coef": t, "every": m}},
                 "mlp": {"kind": "dense", "ff": F, "limit": l}},
                {"type": "delta", "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "conv": K},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": Fs},
                         "router": {"experts": E, "top": k}}},
                {"type": "parallel",
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": c, "bias_max": d,
                                    "q_temp": {"coef": t, "every": m}},
                           "right": {"heads": H, "vdim": Dv, "state": N, "groups": g, "norm_groups": p, "conv": K}},
                 "mlp": null}]}

Tensors (linear weights ``[out, in]``): ``embed`` [V, W], ``final.norm`` [W], with
a loop ``loop.in`` [W, 2 W] and ``loop.step`` [n, W]; per layer i ``l<i>.norm1``
and (with a feed-forward) ``norm2`` [W]; under ``l<i>.mix`` an attention has ``q``
[H D, W], ``q.b``, ``k`` [G D, W], ``k.b``, ``q.norm``, ``k.norm`` [D], ``o`` [W, H D];
a delta has ``q``, ``k`` [G D, W], ``v`` [H Dv, W], ``q.conv``, ``k.conv``, ``v.conv``
[channels, K], ``b``, ``a`` [H, W], ``A_log``, ``dt_bias`` [H], ``g`` [H Dv, W],
``norm`` [Dv], ``o`` [W, H Dv]; a parallel has, under ``left``, an attention's
tensors without the norms, ``rel`` [B, H] (B is the tensor's own; ``bias_rows``
names it where a model is made, not read), ``o.b`` [W] and ``out`` [W], and
under ``right`` ``in`` [2 H Dv + 2 g N + H, W], ``conv`` [H Dv + 2 g N, K], ``conv.b``,
``dt_bias``, ``A_log``, ``D`` [H], ``norm`` [H Dv], ``o`` [W, H Dv] and ``out`` [W].
Under ``l<i>.mlp`` a dense feed-forward has ``gate``, ``up`` [F, W], ``down`` [W, F]; a
moe has ``e<j>.up`` [F, W], ``e<j>.down`` [W, F], ``router`` [E, W], ``router.b`` [E] and,
with a shared expert, ``shared.up`` [Fs, W], ``shared.down`` [W, Fs].
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .mekazen import MAX_POSITIONS, _count, _number, _object
from .qwen3 import ConfigError
from .sadosun import _positive
from .spec import LayerRun, LayerSpec, ModelSpec, PartSpec


def _heads(raw: Mapping[str, Any], where: str) -> Tuple[int, int]:
    heads = _count(raw, "heads", where)
    kv_heads = _count(raw, "kv_heads", where) if raw.get("kv_heads") is not None else heads
    if heads % kv_heads:
        raise ConfigError("InvalidGroupedQueryLayout", f"{where}: {heads} heads over {kv_heads} groups of keys")
    return heads, kv_heads


@dataclass(frozen=True)
class KeyValueAttention:
    """Both attentions of the design: ``bias_max`` None is the one with head norms."""

    heads: int
    kv_heads: int
    dim: int
    scale: float
    q_temp: Optional[Tuple[float, float]]      # (coef, every)
    bias_max: Optional[float] = None           # the distance from which on one bias serves all
    bias_rows: Optional[int] = None            # None: whatever the checkpoint's tensor has

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str, biased: bool = False) -> "KeyValueAttention":
        raw = _object(raw, where)
        heads, kv_heads = _heads(raw, where)
        dim = _count(raw, "dim", where)
        if dim % 2:
            raise ConfigError("OddHeadDimension", f"{where}.dim {dim}")
        if raw.get("vdim", dim) != dim:     # the values are the keys
            raise ConfigError("InvalidValueWidth", f"{where}.vdim {raw.get('vdim')!r} must equal dim {dim}")
        temp = None
        if raw.get("q_temp") is not None:
            given = _object(raw["q_temp"], f"{where}.q_temp")
            temp = (_number(given, "coef", f"{where}.q_temp"), _positive(given, "every", f"{where}.q_temp"))
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, scale=_positive(raw, "scale", where), q_temp=temp,
                   bias_max=_positive(raw, "bias_max", where) if biased else None,
                   bias_rows=_count(raw, "bias_rows", where) if biased and raw.get("bias_rows") is not None else None)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {}
        if self.bias_max is not None:
            out["bias_max"] = self.bias_max
            if self.bias_rows is not None:
                out["bias_rows"] = self.bias_rows
        out.update(dim=self.dim, heads=self.heads, kv_heads=self.kv_heads)
        if self.q_temp is not None:
            out["q_temp"] = {"coef": self.q_temp[0], "every": self.q_temp[1]}
        out.update(scale=self.scale, vdim=self.dim)
        return out

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        q, k = self.heads * self.dim, self.kv_heads * self.dim
        shapes = {f"{base}.q": (q, w), f"{base}.q.b": (q,), f"{base}.k": (k, w), f"{base}.k.b": (k,)}
        if self.bias_max is None:
            shapes.update({f"{base}.q.norm": (self.dim,), f"{base}.k.norm": (self.dim,), f"{base}.o": (w, q)})
        else:
            shapes.update({f"{base}.rel": (self.bias_rows, self.heads), f"{base}.o": (w, q), f"{base}.o.b": (w,)})
        return shapes

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        normed = self.bias_max is None
        norm = lambda name: PartSpec("rmsnorm", {"size": self.dim, "eps": eps, "weight": name}) if normed else None
        return PartSpec("gqa_attention", {
            "hidden_size": w, "num_heads": self.heads, "num_kv_heads": self.kv_heads, "head_dim": self.dim,
            "value_dim": self.dim, "scale": self.scale, "softcap": None, "window": None, "chunk": None,
            "q_proj": f"{base}.q", "k_proj": f"{base}.k", "v_proj": None, "gate_proj": None, "o_proj": f"{base}.o",
            "q_bias": f"{base}.q.b", "k_bias": f"{base}.k.b", "v_bias": None, "shared_kv": False, "qk_norm_scope": "head",
            "q_norm": norm(f"{base}.q.norm"), "k_norm": norm(f"{base}.k.norm"), "position": None, "value_position": None,
            "sink": None, "out_bias": None if normed else f"{base}.o.b",
            "query_factors": PartSpec("log_temperature", {"coef": self.q_temp[0], "every": self.q_temp[1]})
            if self.q_temp is not None else None,
            "distance_bias": None if normed else {"weight": f"{base}.rel", "far": self.bias_max}})


@dataclass(frozen=True)
class HeadDeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "HeadDeltaMixer":
        raw = _object(raw, where)
        heads, kv_heads = _heads(raw, where)
        dim = _count(raw, "dim", where)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim,
                   vdim=_count(raw, "vdim", where) if raw.get("vdim") is not None else dim, conv=_count(raw, "conv", where))

    def to_dict(self) -> Dict[str, Any]:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        return {f"{base}.q": (qk, w), f"{base}.q.conv": (qk, self.conv), f"{base}.k": (qk, w),
                f"{base}.k.conv": (qk, self.conv), f"{base}.v": (v, w), f"{base}.v.conv": (v, self.conv),
                f"{base}.b": (self.heads, w), f"{base}.A_log": (self.heads,), f"{base}.norm": (self.vdim,),
                f"{base}.a": (self.heads, w), f"{base}.dt_bias": (self.heads,), f"{base}.g": (v, w), f"{base}.o": (w, v)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        return PartSpec("head_delta", {
            "hidden_size": w, "num_heads": self.heads, "num_kv_heads": self.kv_heads, "head_dim": self.dim,
            "value_dim": self.vdim, "conv_taps": self.conv, "eps": eps, "q_proj": f"{base}.q", "k_proj": f"{base}.k",
            "v_proj": f"{base}.v", "q_conv": f"{base}.q.conv", "k_conv": f"{base}.k.conv", "v_conv": f"{base}.v.conv",
            "beta_proj": f"{base}.b", "step_proj": f"{base}.a", "step_bias": f"{base}.dt_bias", "a_log": f"{base}.A_log",
            "gate_proj": f"{base}.g", "norm": f"{base}.norm", "o_proj": f"{base}.o"})


@dataclass(frozen=True)
class DualMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "DualMixer":
        raw = _object(raw, where)
        optional = lambda key: _count(raw, key, where) if raw.get(key) is not None else 1
        made = cls(heads=_count(raw, "heads", where), vdim=_count(raw, "vdim", where), state=_count(raw, "state", where),
                   groups=optional("groups"), norm_groups=optional("norm_groups"), conv=_count(raw, "conv", where))
        if made.heads % made.groups or (made.heads * made.vdim) % made.norm_groups:
            raise ConfigError("InvalidGroupedQueryLayout", f"{where}: {made.heads} heads of {made.vdim} values in "
                              f"{made.groups} groups, normed in {made.norm_groups} parts")
        return made

    def to_dict(self) -> Dict[str, Any]:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups,
                "state": self.state, "vdim": self.vdim}

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        inner, pair = self.heads * self.vdim, 2 * self.groups * self.state
        return {f"{base}.in": (2 * inner + pair + self.heads, w), f"{base}.conv": (inner + pair, self.conv),
                f"{base}.conv.b": (inner + pair,), f"{base}.dt_bias": (self.heads,), f"{base}.A_log": (self.heads,),
                f"{base}.D": (self.heads,), f"{base}.norm": (inner,), f"{base}.o": (w, inner)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        return PartSpec("state_space_dual", {
            "hidden_size": w, "num_heads": self.heads, "value_dim": self.vdim, "state_size": self.state,
            "groups": self.groups, "norm_groups": self.norm_groups, "conv_taps": self.conv, "eps": eps,
            "in_proj": f"{base}.in", "conv_weight": f"{base}.conv", "conv_bias": f"{base}.conv.b",
            "step_bias": f"{base}.dt_bias", "a_log": f"{base}.A_log", "skip": f"{base}.D", "norm": f"{base}.norm",
            "o_proj": f"{base}.o"})


@dataclass(frozen=True)
class PairMixer:
    left: KeyValueAttention
    right: DualMixer

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "PairMixer":
        raw = _object(raw, where)
        return cls(left=KeyValueAttention.from_dict(raw.get("left"), f"{where}.left", biased=True),
                   right=DualMixer.from_dict(raw.get("right"), f"{where}.right"))

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        return {**self.left.shapes(f"{base}.left", w), **self.right.shapes(f"{base}.right", w),
                f"{base}.left.out": (w,), f"{base}.right.out": (w,)}

    def part(self, base: str, w: int, eps: float) -> PartSpec:
        norm = lambda name: PartSpec("rmsnorm", {"size": w, "eps": eps, "weight": name})
        return PartSpec("parallel_mixers", {
            "left": self.left.part(f"{base}.left", w, eps), "right": self.right.part(f"{base}.right", w, eps),
            "left_scale": 0.5, "right_scale": 0.5, "left_norm": norm(f"{base}.left.out"),
            "right_norm": norm(f"{base}.right.out")})


_MIXERS = {"attention": KeyValueAttention, "delta": HeadDeltaMixer, "parallel": PairMixer}


@dataclass(frozen=True)
class ClampedDense:
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "kind": "dense", "limit": self.limit}

    def shapes(self, base: str, w: int) -> Dict[str, tuple]:
        return {f"{base}.gate": (self.ff, w), f"{base}.up": (self.ff, w), f"{base}.down": (w, self.ff)}

    def part(self, base: str, w: int) -> PartSpec:
        return PartSpec("swiglu", {"hidden_size": w, "intermediate_size": self.ff, "gate_proj": f"{base}.gate",
                                   "up_proj": f"{base}.up", "down_proj": f"{base}.down", "activation": "clamped",
                                   "limit": self.limit})


@dataclass(frozen=True)
class ChosenExperts:
    ff: int
    experts: int
    top: int
    shared_ff: int          # 0: no expert that every token uses

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "ChosenExperts":
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
        shapes.update({f"{base}.router": (self.experts, w), f"{base}.router.b": (self.experts,)})
        if self.shared_ff:
            shapes.update({f"{base}.shared.up": (self.shared_ff, w), f"{base}.shared.down": (w, self.shared_ff)})
        return shapes

    def part(self, base: str, w: int) -> PartSpec:
        shared = PartSpec("dense_ff", {"hidden_size": w, "intermediate_size": self.shared_ff, "activation": "relu_squared",
                                       "up_proj": f"{base}.shared.up", "down_proj": f"{base}.shared.down"})
        return PartSpec("routed_experts", {
            "hidden_size": w, "intermediate_size": self.ff, "experts": self.experts, "identity": 0, "top": self.top,
            "activation": "relu_squared", "scores": "chosen", "up_proj": base + ".e{}.up", "down_proj": base + ".e{}.down",
            "router": f"{base}.router", "logit_bias": f"{base}.router.b", "shared": shared if self.shared_ff else None})


def _feed_forward(raw: Mapping[str, Any], where: str):
    raw = _object(raw, where)
    kind = raw.get("kind")
    if kind == "dense":
        return ClampedDense(ff=_count(raw, "ff", where), limit=_positive(raw, "limit", where))
    if kind == "moe":
        return ChosenExperts.from_dict(raw, where)
    raise ConfigError("UnsupportedFeedForward", f"{where}.kind {kind!r}; 'dense' or 'moe'")


@dataclass(frozen=True)
class KokolornLayer:
    kind: str
    mixer: object
    mlp: Optional[object]       # None: no feed-forward

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "KokolornLayer":
        raw = _object(raw, where)
        kind = raw.get("type")
        if kind not in _MIXERS:
            raise ConfigError("UnsupportedLayerType", f"{where}.type {kind!r}; this design has {sorted(_MIXERS)}")
        mlp = _feed_forward(raw["mlp"], f"{where}.mlp") if raw.get("mlp") is not None else None
        return cls(kind=kind, mixer=_MIXERS[kind].from_dict(raw.get("mixer"), f"{where}.mixer"), mlp=mlp)

    def to_dict(self) -> Dict[str, Any]:
        return {"mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None,
                "type": self.kind}


@dataclass(frozen=True)
class KokolornConfig:
    """Sizes and constants of one Kokolorn checkpoint."""

    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[KokolornLayer, ...]
    embedding_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    eos_token_ids: tuple = ()

    ARCHITECTURE = "Kokolorn"
    MODEL_TYPE = "kokolorn"

    @classmethod
    def parse(cls, text: str) -> "KokolornConfig":
        try:
            raw = json.loads(text)
        except json.JSONDecodeError as error:
            raise ConfigError("Json", str(error)) from None
        return cls.from_dict(_object(raw, "config.json"))

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KokolornConfig":
        if raw.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError("UnsupportedModelType", f"architecture {raw.get('architecture')!r}")
        vocab, width = _count(raw, "vocab", "config"), _count(raw, "width", "config")
        if width % 8:
            raise ConfigError("MissingDimension", f"width {width} must be a multiple of 8")
        eps = _number(_object(raw.get("norm"), "norm"), "eps", "norm")
        if eps <= 0.0:
            raise ConfigError("InvalidRmsNormEpsilon", str(eps))
        scale = 1.0
        if raw.get("embedding") is not None and _object(raw["embedding"], "embedding").get("scale") is not None:
            scale = _positive(raw["embedding"], "scale", "embedding")
        given = raw.get("layers")
        if not isinstance(given, list) or not given:
            raise ConfigError("MissingDimension", "layers must be a list of at least one layer")
        layers = tuple(KokolornLayer.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(given))
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
        return cls(vocab=vocab, width=width, norm_eps=eps, layers=layers, embedding_scale=scale, loop=loop)

    # ------------------------------------------------------------ derived facts
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    def parameter_count(self) -> int:
        return sum(math.prod(shape) for shape in self.tensor_shapes().values() if None not in shape)

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.ARCHITECTURE, "embedding": {"scale": self.embedding_scale},
               "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        out.update({"norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width})
        return out

    # ------------------------------------------------------------- model spec
    def _order(self) -> Tuple[LayerRun, ...]:
        """Layers in the order they run; every pass after the first has cache entries behind all layers' own."""
        count = len(self.layers)
        if self.loop is None:
            return tuple(LayerRun(layer=index) for index in range(count))
        start, stop, times = self.loop
        runs = [LayerRun(layer=index) for index in range(start)]
        for turn in range(times):
            for index in range(start, stop):
                entry = index if turn == 0 else count + (turn - 1) * (stop - start) + index - start
                runs.append(LayerRun(layer=index, cache=entry, join=0 if index == start else None, turn=turn))
        return tuple(runs + [LayerRun(layer=index) for index in range(stop, count)])

    def to_model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps
        norm = lambda name: PartSpec("rmsnorm", {"size": w, "eps": eps, "weight": name, "one_plus": True})
        layers = []
        for index, layer in enumerate(self.layers):
            base = f"l{index}"
            layers.append(LayerSpec(
                name=base, block=PartSpec("prenorm_residual", {"hidden_size": w}),
                mixer=layer.mixer.part(f"{base}.mix", w, eps),
                feed_forward=layer.mlp.part(f"{base}.mlp", w) if layer.mlp is not None else None,
                mixer_norm=norm(f"{base}.norm1"),
                feed_forward_norm=norm(f"{base}.norm2") if layer.mlp is not None else None))
        joins = () if self.loop is None else (
            PartSpec("mix_first", {"hidden_size": w, "weight": "loop.in", "steps": "loop.step", "turns": self.loop[2]}),)
        spec = ModelSpec(
            architecture=self.ARCHITECTURE, hidden_size=w, vocab_size=self.vocab, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": w, "weight": "embed",
                                                   "scale": self.embedding_scale}),
            layers=tuple(layers), order=self._order(), final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": w, "weight": "embed", "softcap": None}),
            joins=joins)
        spec.validate()
        return spec

    # ------------------------------------------------ tensors of a checkpoint
    def tensor_shapes(self) -> Dict[str, tuple]:
        """Shapes by name; None stands for a size that only the checkpoint's tensor gives."""
        w = self.width
        shapes: Dict[str, tuple] = {"embed": (self.vocab, w)}
        if self.loop is not None:
            shapes.update({"loop.in": (w, 2 * w), "loop.step": (self.loop[2], w)})
        for index, layer in enumerate(self.layers):
            base = f"l{index}"
            shapes[f"{base}.norm1"] = (w,)
            if layer.mlp is not None:
                shapes[f"{base}.norm2"] = (w,)
            shapes.update(layer.mixer.shapes(f"{base}.mix", w))
            if layer.mlp is not None:
                shapes.update(layer.mlp.shapes(f"{base}.mlp", w))
        shapes["final.norm"] = (w,)
        return shapes

    def ignored_tensors(self) -> tuple:
        """The second norm of a layer without a feed-forward, should a checkpoint hold it all the same."""
        return tuple(f"l{index}.norm2" for index, layer in enumerate(self.layers) if layer.mlp is None)

    def norm_tensor(self, name: str):
        """How a tensor of random weights is drawn: False for a matrix
        (N(0, 0.02)); "one" for a factor near 1; "zero" for an offset near 0."""
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "b", "dt_bias", "A_log") and not name.endswith(".mix.b"):
            return "zero"
        if name == "final.norm":
            return "zero"
        if last in ("norm", "out", "D"):     # the plain weights of the norms, and the skip
            return "one"
        return False
