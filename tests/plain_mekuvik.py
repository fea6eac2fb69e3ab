"""A plain, slow implementation of the Mekuvik decoder in numpy.

Whole sequences, no cache, float64, one function per mechanism; the recurrence
hands its state back so that a test can run it in pieces. It shares no code
with ``metallix_b200`` (files are read with the reader of another plain
implementation in this folder). Notation: x is ``[T, W]`` (tokens by width),
positions count from 0, weights are ``[out, in]`` and applied as x @ w.T.
"""
from __future__ import annotations

import math

import numpy as np

from plain_qwen3 import read_model  # noqa: F401  (a reader of config.json + safetensors, nothing else)


# ------------------------------------------------------------ small pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    """z times the standard normal's distribution function."""
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def over_rms(x, eps):
    """x over sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def softmax(scores, visible):
    masked = np.where(visible, scores, -np.inf)
    e = np.where(visible, np.exp(masked - masked.max(axis=-1, keepdims=True)), 0.0)
    return e / e.sum(axis=-1, keepdims=True)


# ----------------------------------------------------------------- positions
def frequencies(rot):
    """(f ``[dims / 2]``, what cos and sin are multiplied by)."""
    dims, base = rot["dims"], rot["base"]
    index = np.arange(dims // 2)
    f = base ** (-2.0 * index / dims)
    stretch = rot.get("scaling")
    if not stretch:
        return f, 1.0
    pair_of = lambda turns: dims * math.log(stretch["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(pair_of(stretch["fast"])), 0)
    hi = min(math.ceil(pair_of(stretch["slow"])), dims - 1)
    ramp = np.clip((index - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / stretch["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(stretch["factor"]) + 1.0


def turn_pairs(x, rot, positions):
    """x ``[T, ..., D]``: the first ``dims`` values in neighbouring pairs, pair i turned by p f_i."""
    f, magnitude = frequencies(rot)
    dims = rot["dims"]
    angle = np.asarray(positions)[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = (np.cos(angle) * magnitude).reshape(shape), (np.sin(angle) * magnitude).reshape(shape)
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---------------------------------------------------------------- attention
def windowed_mask(count, mask):
    """[T, T] (query, key): the last ``size`` positions and the first ``keep_first``."""
    i, j = np.arange(count)[:, None], np.arange(count)[None, :]
    seen = j <= i
    if mask is None:
        return seen
    return seen & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def window_attention(h, tensors, base, mixer, eps, weights_out=None, mask_override=None):
    """Grouped-query attention whose q and k are normed over the whole projection, rotated in
    pairs, in a window beside the first tokens."""
    count, H, D = h.shape[0], mixer["heads"], mixer["dim"]
    G, Dv = mixer.get("kv_heads") or H, mixer.get("vdim") or D
    q = over_rms(h @ tensors[f"{base}.q"].T, eps) * tensors[f"{base}.q.norm"]
    k = over_rms(h @ tensors[f"{base}.k"].T, eps) * tensors[f"{base}.k.norm"]
    v = (h @ tensors[f"{base}.v"].T).reshape(count, G, Dv)
    positions = np.arange(count)
    q, k = q.reshape(count, H, D), k.reshape(count, G, D)
    if mixer.get("rot"):
        q, k = turn_pairs(q, mixer["rot"], positions), turn_pairs(k, mixer["rot"], positions)
    visible = windowed_mask(count, mixer.get("mask") if mask_override is None else mask_override)
    out = np.zeros((count, H, Dv))
    for head in range(H):
        group = head // (H // G)
        p = softmax((q[:, head] @ k[:, group].T) * mixer["scale"], visible)
        if weights_out is not None:
            weights_out.append(p)
        out[:, head] = p @ v[:, group]
    return out.reshape(count, H * Dv) @ tensors[f"{base}.o"].T


def latent_attention(h, tensors, base, mixer, eps, weights_out=None):
    """Keys and values widened from one normed latent per position, one rotated key part for all
    heads, queries through a latent of their own, a gate per value on the heads' output."""
    count, H, D, R = h.shape[0], mixer["heads"], mixer["dim"], mixer["rot_dim"]
    Dv, r = mixer.get("vdim") or D, mixer["kv_rank"]
    positions = np.arange(count)
    cq = over_rms(h @ tensors[f"{base}.dq"].T, eps) * tensors[f"{base}.dq.norm"]
    q = (cq @ tensors[f"{base}.uq"].T).reshape(count, H, D + R)
    down = h @ tensors[f"{base}.dkv"].T
    c = over_rms(down[:, :r], eps) * tensors[f"{base}.dkv.norm"]
    q_far, k_far = q[:, :, D:], down[:, r:]
    if mixer.get("rot"):
        q_far, k_far = turn_pairs(q_far, mixer["rot"], positions), turn_pairs(k_far, mixer["rot"], positions)
    k = (c @ tensors[f"{base}.uk"].T).reshape(count, H, D)
    v = (c @ tensors[f"{base}.uv"].T).reshape(count, H, Dv)
    visible = windowed_mask(count, None)
    out = np.zeros((count, H, Dv))
    for head in range(H):
        scores = (q[:, head, :D] @ k[:, head].T + q_far[:, head] @ k_far.T) * mixer["scale"]
        p = softmax(scores, visible)
        if weights_out is not None:
            weights_out.append(p)
        out[:, head] = p @ v[:, head]
    gated = out.reshape(count, H * Dv) * sigmoid(h @ tensors[f"{base}.g"].T)
    return gated @ tensors[f"{base}.o"].T


# ------------------------------------------------------------ the recurrence
def fading_memory(q, k, v, decay, state=None):
    """One head. q, k ``[T, D]``, v ``[T, Dv]``, one decay: S <- decay S + k v^T, o = S^T q.
    Returns o ``[T, Dv]`` and the last S ``[D, Dv]``."""
    s = np.zeros((q.shape[1], v.shape[1])) if state is None else np.array(state, dtype=np.float64, copy=True)
    out = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        s = decay * s + np.outer(k[t], v[t])
        out[t] = s.T @ q[t]
    return out, s


def lightning(h, tensors, base, mixer, eps, states=None):
    """Linear attention with a fixed decay per head. ``states`` [H of (D, Dv)] come from an earlier
    piece; returns the output and the new states."""
    count, H, D = h.shape[0], mixer["heads"], mixer["dim"]
    Dv = mixer.get("vdim") or D
    q = silu(h @ tensors[f"{base}.q"].T).reshape(count, H, D)
    k = silu(h @ tensors[f"{base}.k"].T).reshape(count, H, D)
    v = silu(h @ tensors[f"{base}.v"].T).reshape(count, H, Dv)
    out, last = np.zeros((count, H, Dv)), []
    for head in range(H):
        o, s = fading_memory(q[:, head], k[:, head], v[:, head], mixer["decay"][head],
                             states[head] if states is not None else None)
        out[:, head] = o
        last.append(s)
    normed = over_rms(out.reshape(count, H * Dv), eps) * tensors[f"{base}.norm"]
    return (normed * sigmoid(h @ tensors[f"{base}.g"].T)) @ tensors[f"{base}.o"].T, last


# ------------------------------------------------------------- feed-forward
def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def gelu_ff(h, up, down):
    return gelu(h @ up.T) @ down.T


def choose_experts(logits, top):
    """The ``top`` largest sigmoid scores (the lower index wins a tie) and these scores as they are."""
    scores = sigmoid(logits)
    chosen = np.argsort(-logits, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(scores, chosen, axis=-1)


def expert_mixture(h, tensors, base, mlp, chosen_out=None):
    """The sum of the chosen experts of the weighted input, and a shared expert's of the plain one."""
    chosen, weights = choose_experts(h @ tensors[f"{base}.router"].T, mlp["router"]["top"])
    if chosen_out is not None:
        chosen_out.append(chosen)
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += gelu_ff(h[rows] * weights[rows, place][:, None], tensors[f"{base}.e{e}.up"],
                                 tensors[f"{base}.e{e}.down"])
    if mlp.get("shared"):
        out += gelu_ff(h, tensors[f"{base}.shared.up"], tensors[f"{base}.shared.down"])
    return out


def feed_forward(h, tensors, base, mlp, chosen_out=None):
    if mlp["kind"] == "dense":
        return gated_ff(h, tensors[f"{base}.gate"], tensors[f"{base}.up"], tensors[f"{base}.down"])
    if mlp["kind"] == "moe":
        return expert_mixture(h, tensors, base, mlp, chosen_out)
    raise ValueError(mlp["kind"])


# ------------------------------------------------------------------ the model
def layer_runs(config):
    """[(layer, whether the embedding output joins first)]: the order in which layers run."""
    loop = config.get("loop")
    count = len(config["layers"])
    if not loop:
        return [(index, False) for index in range(count)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    runs = [(index, False) for index in range(start)]
    for turn in range(times):
        runs += [(index, turn > 0 and index == start) for index in range(start, stop)]
    return runs + [(index, False) for index in range(stop, count)]


def forward_logits(config, tensors, ids, taps=None, seen=None):
    """Logits ``[T, vocab]`` of a whole sequence. ``taps`` (a list) takes the
    residual stream after every layer run; ``seen`` (a dict) takes, per run, the
    attention weights or the chosen experts."""
    tensors = {name: np.asarray(t, dtype=np.float64) for name, t in tensors.items()}
    eps = config["norm"]["eps"]
    x0 = tensors["embed"][np.asarray(ids)]
    x = x0
    for run, (index, joins) in enumerate(layer_runs(config)):
        if joins:
            x = x + x0
        layer = config["layers"][index]
        base, mixer, kind = f"l{index}", layer["mixer"], layer["type"]
        h = over_rms(x, eps) * tensors[f"{base}.norm1"]
        weights = [] if seen is not None else None
        if kind == "lightning":
            mixed, _ = lightning(h, tensors, f"{base}.mix", mixer, eps)
        elif kind == "attention":
            mixed = window_attention(h, tensors, f"{base}.mix", mixer, eps, weights_out=weights)
        elif kind == "latent_attention":
            mixed = latent_attention(h, tensors, f"{base}.mix", mixer, eps, weights_out=weights)
        else:
            raise ValueError(kind)
        if seen is not None and weights:
            seen[(run, "attention")] = weights
        fed = 0.0
        if layer.get("mlp") is not None:
            chosen = [] if seen is not None else None
            fed = feed_forward(h, tensors, f"{base}.mlp", layer["mlp"], chosen)
            if seen is not None and chosen:
                seen[(run, "experts")] = chosen[0]
        x = x + (mixed + fed)
        if taps is not None:
            taps.append(x.copy())
    return (over_rms(x, eps) * tensors["final.norm"]) @ tensors["embed"].T * config.get("logit_scale", 1.0)
