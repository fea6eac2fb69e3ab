"""A plain, slow implementation of the Kokolorn decoder in numpy.

Whole sequences, no cache, float64, one function per mechanism; a recurrence
hands its state back so that a test can run it in pieces. It shares no code
with ``metallix_b200`` (files are read with the reader of the other plain
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


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    """x over sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def centred_norm(x, w, eps):
    """The layers' norm: its stored weight lies around zero, the factor is 1 + w."""
    return over_rms(x, eps) * (1.0 + w)


def softmax(scores, visible):
    masked = np.where(visible, scores, -np.inf)
    e = np.where(visible, np.exp(masked - masked.max(axis=-1, keepdims=True)), 0.0)
    return e / e.sum(axis=-1, keepdims=True)


# ---------------------------------------------------------------- attention
def query_temperature(count, temp):
    """[T]: what the query at position p is multiplied by."""
    p = np.arange(count)
    return 1.0 + temp["coef"] * np.log(np.floor((p + 1) / temp["every"]) + 1.0)


def distance_bucket(n, rows, far):
    """The row of a table of ``rows`` rows that distance n reads: its own below
    half the table, then logarithmic up to ``far``, the last row from there on."""
    half = rows // 2
    if n < half:
        return n
    step = math.floor(math.log(n / half) / math.log(far / half) * (rows - half))
    return min(rows - 1, half + step)


def keys_as_values_attention(h, tensors, base, mixer, eps, norms=True, biased_output=False, weights_out=None,
                             use_bias=True, use_temperature=True):
    """Grouped-query attention without a value projection (the values are the
    keys as projected, bias included, ahead of the key norm) and without
    rotation: positions come in through the queries' temperature and, where the
    layer has a table of them, a learned bias per distance and head."""
    count, H, D = h.shape[0], mixer["heads"], mixer["dim"]
    G = mixer.get("kv_heads") or H
    q = (h @ tensors[f"{base}.q"].T + tensors[f"{base}.q.b"]).reshape(count, H, D)
    k = (h @ tensors[f"{base}.k"].T + tensors[f"{base}.k.b"]).reshape(count, G, D)
    v = k
    if norms:
        q = over_rms(q, eps) * tensors[f"{base}.q.norm"]
        k = over_rms(k, eps) * tensors[f"{base}.k.norm"]
    if mixer.get("q_temp") and use_temperature:
        q = q * query_temperature(count, mixer["q_temp"])[:, None, None]
    i, j = np.arange(count)[:, None], np.arange(count)[None, :]
    table = tensors.get(f"{base}.rel") if use_bias else None
    if table is not None:
        rows = table.shape[0]
        row_of = np.asarray([distance_bucket(n, rows, mixer["bias_max"]) for n in range(count)])
        bucket = row_of[np.maximum(i - j, 0)]
    out = np.zeros((count, H, D))
    for head in range(H):
        group = head // (H // G)
        scores = (q[:, head] @ k[:, group].T) * mixer["scale"]
        if table is not None:
            scores = scores + table[bucket, head]
        p = softmax(scores, j <= i)
        if weights_out is not None:
            weights_out.append(p)
        out[:, head] = p @ v[:, group]
    y = out.reshape(count, H * D) @ tensors[f"{base}.o"].T
    return y + tensors[f"{base}.o.b"] if biased_output else y


# --------------------------------------------------------- the recurrences
def causal_conv(x, taps_weight, before=None):
    """x ``[T, C]``, taps_weight ``[C, K]`` whose last column meets the current
    token: y_t = sum_j w[:, j] x_(t - K + 1 + j), zeros before the sequence
    (or ``before`` ``[K - 1, C]``). Returns y and the last K - 1 inputs."""
    count, channels = x.shape
    k = taps_weight.shape[1]
    if before is None:
        before = np.zeros((k - 1, channels))
    padded = np.concatenate([before, x], axis=0)
    y = np.zeros_like(x)
    for j in range(k):
        y += taps_weight[:, j][None, :] * padded[j:j + count]
    return y, padded[count:]


def delta_rule(q, k, v, beta, decay, state=None):
    """One head. q, k ``[T, D]``, v ``[T, Dv]``, beta and decay ``[T]``. Per token:
    S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.
    Returns o ``[T, Dv]`` and the last S ``[D, Dv]``."""
    count, dim = q.shape
    s = np.zeros((dim, v.shape[1])) if state is None else np.array(state, dtype=np.float64, copy=True)
    out = np.zeros((count, v.shape[1]))
    for t in range(count):
        s = decay[t] * s
        u = beta[t] * (v[t] - s.T @ k[t])
        s = s + np.outer(k[t], u)
        out[t] = s.T @ q[t]
    return out, s


def head_delta(h, tensors, base, mixer, eps, carry=None):
    """The gated delta rule with one decay per head. ``carry`` = (conv inputs
    of q, k, v, states [H, D, Dv]) from an earlier piece; returns the output and
    the new carry."""
    count, H, D = h.shape[0], mixer["heads"], mixer["dim"]
    G, Dv = mixer.get("kv_heads") or H, mixer.get("vdim") or D
    before = carry if carry is not None else (None, None, None, [None] * H)
    q, q_in = causal_conv(h @ tensors[f"{base}.q"].T, tensors[f"{base}.q.conv"], before[0])
    k, k_in = causal_conv(h @ tensors[f"{base}.k"].T, tensors[f"{base}.k.conv"], before[1])
    v, v_in = causal_conv(h @ tensors[f"{base}.v"].T, tensors[f"{base}.v.conv"], before[2])
    q, k, v = silu(q).reshape(count, G, D), silu(k).reshape(count, G, D), silu(v).reshape(count, H, Dv)
    unit = lambda x: x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
    q, k = unit(q) * D ** -0.5, unit(k)
    beta = sigmoid(h @ tensors[f"{base}.b"].T)                                            # [T, H]
    decay = np.exp(-np.exp(tensors[f"{base}.A_log"]) * softplus(h @ tensors[f"{base}.a"].T + tensors[f"{base}.dt_bias"]))
    gate = silu(h @ tensors[f"{base}.g"].T).reshape(count, H, Dv)
    out, states = np.zeros((count, H, Dv)), []
    for head in range(H):
        group = head // (H // G)
        o, s = delta_rule(q[:, group], k[:, group], v[:, head], beta[:, head], decay[:, head], before[3][head])
        out[:, head] = over_rms(o, eps) * tensors[f"{base}.norm"] * gate[:, head]
        states.append(s)
    return out.reshape(count, H * Dv) @ tensors[f"{base}.o"].T, (q_in, k_in, v_in, states)


def dual_scan(x, b, c, dt, decay, skip, state=None):
    """One head of the state-space dual. x ``[T, Dv]``, b, c ``[T, N]``, dt and
    decay ``[T]``: S <- decay S + dt b x^T; y = S^T c + skip x. Returns y and the last S ``[N, Dv]``."""
    count = x.shape[0]
    s = np.zeros((b.shape[1], x.shape[1])) if state is None else np.array(state, dtype=np.float64, copy=True)
    out = np.zeros_like(x)
    for t in range(count):
        s = decay[t] * s + dt[t] * np.outer(b[t], x[t])
        out[t] = s.T @ c[t] + skip * x[t]
    return out, s


def state_space_dual(h, tensors, base, mixer, eps, carry=None):
    """Mamba-2. ``carry`` = (conv inputs, states [H, N, Dv]); returns the output and the new carry."""
    count, H, Dv, N = h.shape[0], mixer["heads"], mixer["vdim"], mixer["state"]
    G, P = mixer.get("groups") or 1, mixer.get("norm_groups") or 1
    inner = H * Dv
    before = carry if carry is not None else (None, [None] * H)
    wide = h @ tensors[f"{base}.in"].T
    z, mid, dt = wide[:, :inner], wide[:, inner:2 * inner + 2 * G * N], wide[:, 2 * inner + 2 * G * N:]
    mid, last = causal_conv(mid, tensors[f"{base}.conv"], before[0])
    mid = silu(mid + tensors[f"{base}.conv.b"])
    x = mid[:, :inner].reshape(count, H, Dv)
    b = mid[:, inner:inner + G * N].reshape(count, G, N)
    c = mid[:, inner + G * N:].reshape(count, G, N)
    dt = softplus(dt + tensors[f"{base}.dt_bias"])
    decay = np.exp(-np.exp(tensors[f"{base}.A_log"]) * dt)
    y, states = np.zeros((count, H, Dv)), []
    for head in range(H):
        group = head // (H // G)
        y[:, head], s = dual_scan(x[:, head], b[:, group], c[:, group], dt[:, head], decay[:, head],
                                  tensors[f"{base}.D"][head], before[1][head])
        states.append(s)
    gated = (y.reshape(count, inner) * silu(z)).reshape(count, P, inner // P)
    normed = over_rms(gated, eps).reshape(count, inner) * tensors[f"{base}.norm"]
    return normed @ tensors[f"{base}.o"].T, (last, states)


def side_by_side(h, tensors, base, mixer, eps, weights_out=None, **switches):
    """Half the sum of both mixers' outputs, each over its own root mean square times a weight."""
    left = keys_as_values_attention(h, tensors, f"{base}.left", mixer["left"], eps, norms=False, biased_output=True,
                                    weights_out=weights_out, **switches)
    right, _ = state_space_dual(h, tensors, f"{base}.right", mixer["right"], eps)
    return 0.5 * (over_rms(left, eps) * tensors[f"{base}.left.out"] + over_rms(right, eps) * tensors[f"{base}.right.out"])


# ------------------------------------------------------------- feed-forward
def clamped_ff(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def squared_ff(h, up, down):
    return np.maximum(h @ up.T, 0.0) ** 2 @ down.T


def choose_experts(logits, top):
    """The ``top`` largest logits (the lower index wins a tie), weighted by the softmax over them alone."""
    chosen = np.argsort(-logits, axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(logits, chosen, axis=-1)
    return chosen, softmax(picked, np.ones_like(picked, dtype=bool))


def expert_mixture(h, tensors, base, mlp, chosen_out=None):
    chosen, weights = choose_experts(h @ tensors[f"{base}.router"].T + tensors[f"{base}.router.b"], mlp["router"]["top"])
    if chosen_out is not None:
        chosen_out.append(chosen)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weights[t]):
            out[t] += w * squared_ff(h[t:t + 1], tensors[f"{base}.e{e}.up"], tensors[f"{base}.e{e}.down"])[0]
    if mlp.get("shared"):
        out += squared_ff(h, tensors[f"{base}.shared.up"], tensors[f"{base}.shared.down"])
    return out


def feed_forward(h, tensors, base, mlp, chosen_out=None):
    if mlp["kind"] == "dense":
        return clamped_ff(h, tensors[f"{base}.gate"], tensors[f"{base}.up"], tensors[f"{base}.down"], mlp["limit"])
    if mlp["kind"] == "moe":
        return expert_mixture(h, tensors, base, mlp, chosen_out)
    raise ValueError(mlp["kind"])


# ------------------------------------------------------------------ the model
def layer_runs(config):
    """[(layer, pass or None, first of its pass)]: the order in which layers run."""
    loop = config.get("loop")
    count = len(config["layers"])
    if not loop:
        return [(index, None, False) for index in range(count)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    runs = [(index, None, False) for index in range(start)]
    for turn in range(times):
        runs += [(index, turn, index == start) for index in range(start, stop)]
    return runs + [(index, None, False) for index in range(stop, count)]


def forward_logits(config, tensors, ids, taps=None, seen=None, **switches):
    """Logits ``[T, vocab]`` of a whole sequence. ``taps`` (a list) takes the
    residual stream after every layer run; ``seen`` (a dict) takes, per run, the
    attention weights or the chosen experts."""
    tensors = {name: np.asarray(t, dtype=np.float64) for name, t in tensors.items()}
    eps = config["norm"]["eps"]
    x0 = tensors["embed"][np.asarray(ids)] * (config.get("embedding") or {}).get("scale", 1.0)
    x = x0
    for run, (index, turn, first) in enumerate(layer_runs(config)):
        if first:
            x = np.concatenate([x, x0], axis=1) @ tensors["loop.in"].T + tensors["loop.step"][turn]
        layer = config["layers"][index]
        base, mixer, kind = f"l{index}", layer["mixer"], layer["type"]
        h = centred_norm(x, tensors[f"{base}.norm1"], eps)
        weights = [] if seen is not None else None
        if kind == "attention":
            mixed = keys_as_values_attention(h, tensors, f"{base}.mix", mixer, eps, weights_out=weights, **switches)
        elif kind == "delta":
            mixed, _ = head_delta(h, tensors, f"{base}.mix", mixer, eps)
        elif kind == "parallel":
            mixed = side_by_side(h, tensors, f"{base}.mix", mixer, eps, weights_out=weights, **switches)
        else:
            raise ValueError(kind)
        x = x + mixed
        if seen is not None and weights:
            seen[(run, "attention")] = weights
        if layer.get("mlp") is not None:
            chosen = [] if seen is not None else None
            x = x + feed_forward(centred_norm(x, tensors[f"{base}.norm2"], eps), tensors, f"{base}.mlp", layer["mlp"], chosen)
            if seen is not None and chosen:
                seen[(run, "experts")] = chosen[0]
        if taps is not None:
            taps.append(x.copy())
    return centred_norm(x, tensors["final.norm"], eps) @ tensors["embed"].T
