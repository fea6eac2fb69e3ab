"""The Kokolorn decoder in the engine against the plain implementation
(``plain_kokolorn.py``): its configuration and mechanisms one at a time, then
whole prompts layer run by layer run, decoding through the cache and the state,
portions, mixed batches, pages and slots that come back, keys far back and at
page borders, distances inside and outside the bias table's edges, the first
tokens, long decoding, generation through the scheduler and the trace program.
Every model here is tiny, made for the test with random weights, and differs
from layer to layer."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_kokolorn as plain
import replay_helpers as cuts
from conftest import ROOT, random_ids


# ------------------------------------------------------------ configurations
def attention(heads, kv_heads, dim, scale, temp=None, bias_max=None, rows=None):
    out = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads:
        out["kv_heads"] = kv_heads
    if temp:
        out["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if bias_max:
        out["bias_max"], out["bias_rows"] = bias_max, rows
    return out


def delta(heads, kv_heads, dim, vdim, conv):
    out = {"heads": heads, "dim": dim, "conv": conv}
    if kv_heads:
        out["kv_heads"] = kv_heads
    if vdim:
        out["vdim"] = vdim
    return out


def dual(heads, vdim, state, conv, groups=None, norm_groups=None):
    out = {"heads": heads, "vdim": vdim, "state": state, "conv": conv}
    if groups:
        out["groups"] = groups
    if norm_groups:
        out["norm_groups"] = norm_groups
    return out


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# SMALL: sizes that are no power of two; the loop in the middle of the stack, over a pair of side-by-side mixers and
# a layer without feed-forward; an odd number of bias rows; two groups of B and C, the norm in three parts; a shared
# expert of another width; two heads per query/key group in the recurrence; every expert chosen.
SMALL = {"architecture": "Kokolorn", "vocab": 203, "width": 72, "norm": {"eps": 2e-6}, "embedding": {"scale": 3.5},
         "loop": {"start": 1, "stop": 4, "times": 2},
         "layers": [
             layer("delta", delta(4, 2, 12, 20, 3), dense(40, 0.7)),
             layer("parallel", {"left": attention(4, 2, 16, 0.3, (0.4, 9), 23, 13), "right": dual(6, 10, 14, 3, 2, 3)},
                   moe(24, 5, 2, 40)),
             layer("attention", attention(3, 1, 10, 0.35, (0.6, 5)), None),
             layer("delta", delta(3, 0, 8, 6, 2), moe(16, 3, 3)),
             layer("attention", attention(4, 4, 18, 0.2, (0.25, 16)), moe(20, 7, 1, 16))]}
# WIDE: heads of 64 and 128 values (the tensor-core kernels' sizes) with two and eight query heads per key head, a
# bias table that reaches over several key tiles and one that ends inside a tile, a recurrence with one query/key
# group for four heads, a state-space mixer with 128 states and heads of 64 values, the first layers looped.
WIDE = {"architecture": "Kokolorn", "vocab": 310, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 6.0},
        "loop": {"start": 0, "stop": 1, "times": 3},
        "layers": [
            layer("attention", attention(4, 2, 64, 0.11, (0.5, 50)), moe(32, 6, 2, 32)),
            layer("parallel", {"left": attention(8, 1, 64, 0.09, (0.3, 128), 300, 16), "right": dual(4, 64, 128, 4, 1, 2)},
                  dense(192, 1.5)),
            layer("delta", delta(4, 1, 64, 48, 4), moe(64, 4, 1)),
            layer("parallel", {"left": attention(2, 1, 128, 0.07, None, 70, 8), "right": dual(2, 32, 16, 2)}, None)]}
# BARE: the switches' other position: no loop, no scale of the embedding, no temperature, a key head per query head,
# one expert of which one is chosen, convolutions of one tap, a bias table of two rows, a state of one value.
BARE = {"architecture": "Kokolorn", "vocab": 99, "width": 48, "norm": {"eps": 1e-5},
        "layers": [
            layer("attention", attention(2, 0, 8, 0.5), moe(20, 1, 1)),
            layer("delta", delta(1, 0, 5, 0, 1), None),
            layer("parallel", {"left": attention(3, 0, 6, 0.4, None, 2, 2), "right": dual(1, 7, 1, 1)}, dense(24, 0.5))]}
MODELS = {"small": (SMALL, 51, 8, 1.0), "wide": (WIDE, 52, 16, 1.0), "bare": (BARE, 53, 4, 1.0),
          # score scales four times as large: which keys a query looks at decides its output
          "sharp": (SMALL, 54, 8, 4.0)}
CASES = [(name, dtype) for name in MODELS for dtype in ("float32", "bfloat16") if (name, dtype) != ("sharp", "bfloat16")]
TOL = {"float32": 2e-4, "bfloat16": 3e-1}
TOL_SHARP = 1e-3


def bound(name, dtype):
    return TOL_SHARP if name == "sharp" else TOL[dtype]


def compare_replay(name, dtype, seen, reference):
    """float32: every position within the bound. bfloat16: a router's close
    call may go the other way at a position or two, so the bound holds for 19
    positions out of 20, the median lies well inside it, and at most one
    position in fifty is off by the size of a logit; a lost state or a wrong
    key would put every position behind it there."""
    errors = np.asarray([float(np.abs(row - reference[key][at]).max()) for (key, at), row in seen.items()])
    assert len(errors)
    if dtype == "float32":
        assert errors.max() < bound(name, dtype), errors.max()
    else:
        assert np.median(errors) < 0.4 * TOL[dtype] and np.quantile(errors, 0.95) < TOL[dtype] \
            and (errors > 1.5).mean() <= 0.02, (np.median(errors), np.quantile(errors, 0.95), (errors > 1.5).mean())


def sharpened(raw, factor):
    raw = json.loads(json.dumps(raw))
    for spec in raw["layers"]:
        if spec["type"] == "attention":
            spec["mixer"]["scale"] *= factor
        elif spec["type"] == "parallel":
            spec["mixer"]["left"]["scale"] *= factor
    return raw


def write_folder(folder, raw, seed, sharpen):
    """config.json + model.safetensors: bfloat16 matrices, float32 vectors (so
    that the engine and the plain side hold the same values). Projections are
    larger than the generator's (0.02) so that scores, gates and states move;
    step sizes are small so that the state reaches far back; biases and the
    distances' numbers are of the size of the scores."""
    from metallix_b200.config import KokolornConfig
    from metallix_b200.weights import random_tensors
    from metallix_b200.weights.safetensors_io import write_file
    config = KokolornConfig.from_dict(sharpened(raw, sharpen))
    tensors = random_tensors(config, seed, dtype="bfloat16", norm_dtype="float32")
    for name, value in tensors.items():
        last = name.rsplit(".", 1)[-1]
        if last == "conv":
            tensors[name] = (value.float() * 15.0).to(torch.bfloat16)
        elif last == "rel":
            tensors[name] = (value.float() * 60.0).to(torch.bfloat16)
        elif name == "loop.step":
            tensors[name] = (value.float() * 30.0).to(torch.bfloat16)
        elif last == "dt_bias":
            tensors[name] = value - 3.0
        elif last == "b" and value.dim() == 1:
            tensors[name] = value * 5.0
        elif value.dim() == 2:
            tensors[name] = (value.float() * (8.0 if name == "embed" else 4.0)).to(torch.bfloat16)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(config.to_dict(), handle)
    write_file(os.path.join(folder, "model.safetensors"), {k: v.cpu() for k, v in tensors.items()},
               order=list(config.tensor_shapes()))
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """name -> (folder, config dict, tensors as float64 numpy, page size)."""
    out = {}
    for name, (raw, seed, page, sharpen) in MODELS.items():
        folder = write_folder(str(tmp_path_factory.mktemp(f"kokolorn_{name}")), raw, seed, sharpen)
        config, tensors = plain.read_model(folder)
        out[name] = (folder, config, tensors, page)
    return out


def make_engine(folders, name, dtype, pages=96, **options):
    from metallix_b200.engine import Engine
    folder, _, _, page = folders[name]
    return Engine.from_folder(folder, dtype=dtype, page_tokens=page, num_pages=pages,
                              max_requests=options.pop("max_requests", 8), **options)


def reference_logits(folders, name, requests):
    _, config, tensors, _ = folders[name]
    return {key: plain.forward_logits(config, tensors, ids) for key, ids in requests.items()}


def some_requests(name, seed, lengths):
    vocab = MODELS[name][0]["vocab"]
    return {f"r{n}": random_ids(seed + n, length, vocab) for n, length in enumerate(lengths)}


# ------------------------------------------------ configuration (no GPU needed)
def test_configuration_round_trip_and_registry():
    from metallix_b200.config import ConfigError, KokolornConfig, parse_config, resolve
    for raw in (SMALL, WIDE, BARE):
        config = parse_config(raw)
        assert isinstance(config, KokolornConfig) and resolve(raw).kind == "kokolorn"
        assert KokolornConfig.from_dict(config.to_dict()) == config
        assert json.loads(json.dumps(config.to_dict())) == config.to_dict()
        shapes, w = config.tensor_shapes(), raw["width"]
        assert shapes["embed"] == (raw["vocab"], w) and shapes["final.norm"] == (w,) and "head" not in shapes
        loop = raw.get("loop")
        assert ("loop.in" in shapes) == ("loop.step" in shapes) == (loop is not None)
        for index, spec in enumerate(raw["layers"]):
            base, mixer = f"l{index}", spec["mixer"]
            assert shapes[f"{base}.norm1"] == (w,) and (f"{base}.norm2" in shapes) == (spec["mlp"] is not None)
            if spec["type"] == "delta":
                heads = mixer["heads"]
                groups, vdim = mixer.get("kv_heads") or heads, mixer.get("vdim") or mixer["dim"]
                assert shapes[f"{base}.mix.q"] == shapes[f"{base}.mix.k"] == (groups * mixer["dim"], w)
                assert shapes[f"{base}.mix.v.conv"] == (heads * vdim, mixer["conv"]) and shapes[f"{base}.mix.norm"] == (vdim,)
                assert shapes[f"{base}.mix.a"] == shapes[f"{base}.mix.b"] == (heads, w) and shapes[f"{base}.mix.g"] == (heads * vdim, w)
            elif spec["type"] == "attention":
                kv = mixer.get("kv_heads") or mixer["heads"]
                assert shapes[f"{base}.mix.k"] == (kv * mixer["dim"], w) and shapes[f"{base}.mix.k.norm"] == (mixer["dim"],)
                assert f"{base}.mix.v" not in shapes and f"{base}.mix.rel" not in shapes and f"{base}.mix.o.b" not in shapes
            else:
                left, right = mixer["left"], mixer["right"]
                inner, pair = right["heads"] * right["vdim"], 2 * right.get("groups", 1) * right["state"]
                assert shapes[f"{base}.mix.left.rel"] == (left["bias_rows"], left["heads"])
                assert shapes[f"{base}.mix.left.o.b"] == shapes[f"{base}.mix.right.out"] == (w,)
                assert f"{base}.mix.left.q.norm" not in shapes
                assert shapes[f"{base}.mix.right.in"] == (2 * inner + pair + right["heads"], w)
                assert shapes[f"{base}.mix.right.conv"] == (inner + pair, right["conv"])
            if spec["mlp"] is not None and spec["mlp"]["kind"] == "moe":
                count = spec["mlp"]["router"]["experts"]
                assert shapes[f"{base}.mlp.router"] == (count, w) and shapes[f"{base}.mlp.router.b"] == (count,)
                assert (f"{base}.mlp.shared.up" in shapes) == ("shared" in spec["mlp"]) and f"{base}.mlp.e0.gate" not in shapes
        model = config.to_model_spec()
        want = [(index, turn if turn is not None else 0, first) for index, turn, first in plain.layer_runs(raw)]
        assert [(run.layer, run.turn, run.join == 0) for run in model.order] == want
        entries = [run.cache_entry() for run in model.order]
        assert len(set(entries)) == len(entries) and sorted(entries) == list(range(len(entries)))   # each pass its own
        assert all(run.write_cache for run in model.order)
    open_rows = json.loads(json.dumps(SMALL))
    del open_rows["layers"][1]["mixer"]["left"]["bias_rows"]
    assert parse_config(open_rows).tensor_shapes()["l1.mix.left.rel"] == (None, 4)     # left to the checkpoint's tensor
    refusals = [
        ("UnsupportedLayerType", lambda c: c["layers"][1].update(type="channel_delta")),
        ("InvalidGroupedQueryLayout", lambda c: c["layers"][2]["mixer"].update(kv_heads=2)),
        ("InvalidGroupedQueryLayout", lambda c: c["layers"][0]["mixer"].update(kv_heads=3)),
        ("InvalidGroupedQueryLayout", lambda c: c["layers"][1]["mixer"]["right"].update(groups=4)),
        ("InvalidGroupedQueryLayout", lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7)),
        ("InvalidValueWidth", lambda c: c["layers"][2]["mixer"].update(vdim=8)),
        ("OddHeadDimension", lambda c: c["layers"][2]["mixer"].update(dim=9)),
        ("UnsupportedFeedForward", lambda c: c["layers"][1]["mlp"].update(kind="relu")),
        ("Json", lambda c: c["layers"][1]["mlp"]["router"].update(top=6)),
        ("Json", lambda c: c["layers"][0]["mlp"].update(limit=0.0)),
        ("Json", lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0)),
        ("Json", lambda c: c["layers"][1]["mixer"]["left"].update(bias_max=None)),
        ("Json", lambda c: c["layers"][2]["mixer"].update(scale=-1.0)),
        ("Json", lambda c: c["loop"].update(stop=6)),
        ("Json", lambda c: c["loop"].update(start=4)),
        ("Json", lambda c: c["loop"].update(start=-1)),
        ("MissingDimension", lambda c: c["loop"].update(times=0)),
        ("MissingDimension", lambda c: c.update(width=70)),
        ("InvalidRmsNormEpsilon", lambda c: c["norm"].update(eps=0.0)),
        ("MissingDimension", lambda c: c.update(layers=[]))]
    for kind, change in refusals:
        raw = json.loads(json.dumps(SMALL))
        change(raw)
        with pytest.raises(ConfigError) as caught:
            parse_config(raw)
        assert caught.value.kind == kind, (kind, caught.value.kind)


def test_random_weights_and_sizes_left_to_the_checkpoint(tmp_path):
    from metallix_b200.config import KokolornConfig
    from metallix_b200.weights import CheckpointError, load_tensors, random_tensors, write_model_folder
    config = KokolornConfig.from_dict(SMALL)
    tensors = random_tensors(config, 3, dtype="float32")
    assert float(tensors["l0.norm1"].abs().max()) <= 0.1 and float(tensors["l1.mix.left.o.b"].abs().max()) <= 0.1
    assert abs(float(tensors["l1.mix.left.out"].mean()) - 1.0) < 0.1 and abs(float(tensors["l2.mix.q.norm"].mean()) - 1.0) < 0.1
    assert abs(float(tensors["l1.mix.right.D"].mean()) - 1.0) < 0.1 and tensors["l0.mix.b"].shape == (4, 72)
    folder = write_model_folder(str(tmp_path / "m"), config, 3)
    assert set(load_tensors(folder, config)) == set(config.tensor_shapes())
    raw = json.loads(json.dumps(SMALL))      # a config.json that does not name the table's rows: the tensor gives them
    del raw["layers"][1]["mixer"]["left"]["bias_rows"]
    unnamed = KokolornConfig.from_dict(raw)
    assert load_tensors(folder, unnamed)["l1.mix.left.rel"].shape == (13, 4)
    with pytest.raises(ValueError):
        random_tensors(unnamed, 3)
    raw["layers"][1]["mixer"]["right"]["state"] = 15
    with pytest.raises(CheckpointError):
        load_tensors(folder, KokolornConfig.from_dict(raw))


def cpu_model(raw):
    from metallix_b200.config import KokolornConfig
    from metallix_b200.engine.model import DecoderModel
    from metallix_b200.parts.registry import Runtime
    from metallix_b200.weights import random_tensors
    config = KokolornConfig.from_dict(raw)
    tensors = random_tensors(config, 1, dtype="float32")
    return DecoderModel(config.to_model_spec(), dict(tensors), Runtime(device=torch.device("cpu"), dtype=torch.float32,
                                                                       max_positions=64)), tensors


def test_cache_needs_tables_and_the_passes_entries():
    """Every pass of a looped layer has an entry of its own with the same
    needs; the bias table is spread over the distances; the temperature is a
    table over positions; a looped layer's weights count once per pass."""
    model, tensors = cpu_model(SMALL)
    needs = model.cache_needs()
    shape = lambda need: [(n.kind, tuple(n.state_shape) if n.kind == "state" else (n.kv_heads, n.head_dim)) for n in need.flat()]
    want = {0: [("state", (4, 20, 12)), ("state", (2, 2 * 2 * 12 + 4 * 20))],
            1: [("kv_pages", (2, 16)), ("state", (6, 10, 14)), ("state", (2, 60 + 2 * 2 * 14))],
            2: [("kv_pages", (1, 10))], 3: [("state", (3, 6, 8)), ("state", (1, 2 * 3 * 8 + 3 * 6))], 4: [("kv_pages", (4, 18))]}
    want.update({5: want[1], 6: want[2], 7: want[3]})
    assert [shape(need) for need in needs] == [want[index] for index in range(8)]
    left = model.blocks[1].mixer.left
    table = tensors["l1.mix.left.rel"].double().numpy()
    for n in range(60):
        row = plain.distance_bucket(n, 13, 23)
        at = min(n, left.distance_bias.shape[1] - 1)
        assert np.allclose(left.distance_bias[:, at].double().numpy(), table[row]), n
    assert left.distance_bias.shape[1] <= 24 and not left.own_values and left.out_bias is not None
    assert np.allclose(left.query_factors.double().numpy(), plain.query_temperature(64, {"coef": 0.4, "every": 9}), atol=1e-6)
    assert model.blocks[2].mixer.distance_bias is None and model.blocks[2].feed_forward is None
    once = dict(SMALL, loop={"start": 1, "stop": 4, "times": 1})
    layers = sum(part.weight_bytes() for block in model.blocks[1:4] for part in (block.mixer, block.feed_forward)
                 if part is not None)
    assert model.weight_bytes() - cpu_model(once)[0].weight_bytes() == layers + model.joins[0].weight_bytes()
    assert cpu_model(BARE)[0].joins == []


def test_rows_of_a_distance_table():
    """The row every distance reads, against the expression itself, for even
    and odd tables and far ends that are no whole number; ends where a
    quotient of logarithms is a whole number belong to the further row."""
    from metallix_b200.parts.attention import distance_rows
    for rows, far in ((32, 200), (32, 128), (16, 100), (5, 9), (2, 3), (33, 1000), (20, 77.5), (64, 3000), (3, 2), (8, 5)):
        got = distance_rows(rows, far)
        assert len(got) <= far + 1 and got[-1] == rows - 1 and got[-2] < rows - 1
        for n in range(int(far) + 20):
            assert got[min(n, len(got) - 1)] == plain.distance_bucket(n, rows, far), (rows, far, n)
    got = distance_rows(32, 256)       # 16 rows over a factor of 16: a doubling every four rows
    assert [got[n] for n in (15, 16, 31, 32, 63, 64, 127, 128)] == [15, 16, 19, 20, 23, 24, 27, 28]
    for rows, far in ((1, 10), (8, 4), (8, 3)):
        with pytest.raises(ValueError):
            distance_rows(rows, far)


def random_model(raw, seed):
    from metallix_b200.config import KokolornConfig
    rng = np.random.default_rng(seed)
    shapes = KokolornConfig.from_dict(raw).tensor_shapes()
    return {name: rng.normal(size=shape) * (0.1 if len(shape) <= 1 else 0.3) for name, shape in shapes.items()}


def test_the_plain_side_in_pieces():
    """The plain implementation itself: logits do not change when more tokens
    follow; both recurrences in pieces, their states and convolutions' inputs
    handed on, equal one run; single steps by hand."""
    rng = np.random.default_rng(0)
    tensors = random_model(SMALL, 0)
    ids = random_ids(1, 30, 203)
    whole = plain.forward_logits(SMALL, tensors, ids)
    assert np.allclose(plain.forward_logits(SMALL, tensors, ids[:19]), whole[:19], atol=1e-9)
    h = rng.normal(size=(25, 72))
    for run in (lambda piece, carry: plain.head_delta(piece, tensors, "l0.mix", SMALL["layers"][0]["mixer"], 1e-6, carry),
                lambda piece, carry: plain.state_space_dual(piece, tensors, "l1.mix.right", SMALL["layers"][1]["mixer"]["right"],
                                                            1e-6, carry)):
        once, _ = run(h, None)
        first, carry = run(h[:2], None)
        second, carry = run(h[2:11], carry)
        third, _ = run(h[11:], carry)
        assert np.allclose(np.concatenate([first, second, third]), once, atol=1e-12)
    q, k, v = np.array([[0.6, 0.8]]), np.array([[1.0, 0.0]]), np.array([[2.0, -1.0, 0.5]])
    out, state = plain.delta_rule(q, k, v, np.array([0.5]), np.array([0.9]))
    assert np.allclose(state, np.outer(k[0], 0.5 * v[0])) and np.allclose(out[0], 0.6 * 0.5 * v[0])
    out, state = plain.delta_rule(q, k, v, np.array([1.0]), np.array([0.5]), state)
    assert np.allclose(state[0], v[0])      # beta 1: the key's row now holds the value whatever it held
    out, state = plain.dual_scan(v, k, q, np.array([2.0]), np.array([0.5]), 3.0, np.ones((2, 3)))
    assert np.allclose(state, 0.5 + np.outer(k[0], 2.0 * v[0])) and np.allclose(out[0], state.T @ q[0] + 3.0 * v[0])
    chosen, weights = plain.choose_experts(np.array([[1.0, 3.0, 2.0, 3.0]]), 2)
    assert chosen[0].tolist() == [1, 3] and np.allclose(weights, 0.5)
    assert np.allclose(plain.query_temperature(7, {"coef": 2.0, "every": 3}), 1.0 + 2.0 * np.log([1, 1, 2, 2, 2, 3, 3]))
    one = np.ones((1, 1))
    assert np.isclose(plain.clamped_ff(5.0 * one, one, one, one, 2.0)[0, 0], 2.0 / (1.0 + np.exp(-3.404)) * 3.0)
    assert np.isclose(plain.clamped_ff(5.0 * one, -one, -one, one, 2.0)[0, 0], -5.0 / (1.0 + np.exp(8.51)) * -1.0)


def test_the_models_of_these_tests_show_a_bias_a_temperature_a_state_and_a_pass(folders):
    """What the tests below can see: on the plain side, scores without the
    distances' biases or with a table one distance longer, queries without
    their temperature, a state lost at one position, one pass fewer and passes
    that do not know which one they are each move the logits by far more than
    the bound the engine is held to."""
    _, config, tensors, _ = folders["sharp"]
    tensors = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    ids = random_ids(40, 75, config["vocab"])
    base = plain.forward_logits(config, tensors, ids)
    longer = json.loads(json.dumps(config))
    longer["layers"][1]["mixer"]["left"]["bias_max"] += 1
    fewer = json.loads(json.dumps(config))
    fewer["loop"]["times"] = 1
    same = dict(tensors, **{"loop.step": np.repeat(tensors["loop.step"][:1], 2, axis=0)})
    lost = np.concatenate([plain.forward_logits(config, tensors, ids[:60]), plain.forward_logits(config, tensors, ids[60:])])
    gap = lambda logits, first=0: np.abs(logits - base)[first:].max()
    gaps = {"bias": gap(plain.forward_logits(config, tensors, ids, use_bias=False)),
            "edge": gap(plain.forward_logits(longer, tensors, ids)),
            "temperature": gap(plain.forward_logits(config, tensors, ids, use_temperature=False)),
            "state": gap(lost, 60), "passes": gap(plain.forward_logits(fewer, dict(tensors), ids)),
            "step": gap(plain.forward_logits(config, same, ids))}
    assert min(gaps.values()) > 30 * TOL_SHARP, gaps


# --------------------------------------------------------- mechanisms alone
gpu = pytest.mark.gpu


def dev(array, dtype=torch.float32):
    return torch.tensor(np.asarray(array), dtype=dtype, device="cuda")


def rounded(array, dtype):
    return torch.tensor(np.asarray(array), dtype=dtype).double().numpy()


def rows_of(lengths):
    starts, cursor = [], 0
    for length in lengths:
        starts.append(cursor)
        cursor += length
    return starts


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["delta", "dual"])
@pytest.mark.parametrize("heads, groups, dim, vdim", [(4, 2, 12, 20), (2, 2, 40, 8), (1, 1, 5, 5), (4, 1, 64, 128), (3, 3, 128, 72),
                                                      (2, 1, 200, 33), (1, 1, 1, 3)])
def test_recurrences_with_one_decay_per_head(dtype, kind, heads, groups, dim, vdim):
    """The delta rule with one decay per head and the state-space dual over
    request rows of unequal length in one launch (a single token, a padding
    row), continued twice from the state the launch before left, against the
    plain recurrence in one piece. Decays are slow, the first token's value is
    large and the last token's query is the first token's key, so that what the
    first token wrote is what the last one reads."""
    from metallix_b200 import ops
    rng = np.random.default_rng(heads * dim + vdim)
    pieces = [[23, 1, 0, 5], [1, 1, 0, 40], [9, 3, 0, 1]]
    slots = [2, 0, 1, 3]
    totals = [sum(p[row] for p in pieces) for row in range(4)]
    rate = rounded(np.exp(rng.normal(size=heads) * 0.3), torch.float32)
    bias = rounded(rng.normal(size=heads) * 0.5 - 4.0, torch.float32)
    skip = rounded(rng.normal(size=heads), torch.float32)
    seq = []
    for total in totals:
        first = np.where(np.arange(total) == 0, 64.0, 1.0)[:, None]
        q_rows, k_rows = rng.normal(size=(total, groups * dim)), rng.normal(size=(total, groups * dim))
        if total > 30:
            q_rows[-1] = k_rows[0]
        seq.append({"q": rounded(q_rows, dtype), "k": rounded(k_rows, dtype),
                    "v": rounded(rng.normal(size=(total, heads * vdim)) * first, dtype),
                    "b": rounded(rng.normal(size=(total, heads)) * 2.0, dtype),
                    "s": rounded(rng.normal(size=(total, heads)), dtype)})
    state = torch.full((5, heads, vdim, dim), 3.0, device="cuda")      # S transposed: a column's channels side by side
    for slot in slots:
        state[slot].zero_()
    got = [[] for _ in totals]
    done = [0] * 4
    for lengths in pieces:
        starts = rows_of(lengths)
        pack = lambda key: np.concatenate([seq[row][key][done[row]:done[row] + n] for row, n in enumerate(lengths)])
        wide = dev(np.concatenate([np.zeros((sum(lengths), 8)), pack("q"), pack("k"), pack("v"), pack("b"), pack("s"),
                                   np.zeros((sum(lengths), 3))], axis=1), dtype)
        at = 8 + 2 * groups * dim + heads * vdim
        where = (8, 8 + groups * dim, 8 + 2 * groups * dim)
        row_lists = (dev(starts, torch.int32), dev(lengths, torch.int32), dev(slots, torch.int32))
        beta, step = wide[:, at:at + heads], wide[:, at + heads:at + 2 * heads]
        if kind == "delta":
            out = ops.delta_rule(wide, where, beta, step, dev(bias), dev(rate), state, *row_lists, heads, groups, dim, vdim,
                                 decay="head", longest=max(lengths))
        else:
            out = ops.state_space_dual(wide, where, step, dev(bias), dev(rate), dev(skip), state, *row_lists, heads, groups, dim,
                                       vdim, longest=max(lengths))
        ops.check_status("cuda")
        for row, n in enumerate(lengths):
            got[row].append(out[starts[row]:starts[row] + n].double().cpu().numpy())
            done[row] += n
    assert float(state[4].min()) == 3.0 and float(state[1].abs().max()) == 0.0      # an untouched slot, a padding row's slot
    unit = lambda x: x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
    for row, total in enumerate(totals):
        if not total:
            continue
        s = seq[row]
        q, k = s["q"].reshape(total, groups, dim), s["k"].reshape(total, groups, dim)
        step = plain.softplus(s["s"] + bias)
        decay = np.exp(-rate[None, :] * step)
        for head in range(heads):
            group, v = head // (heads // groups), s["v"][:, head * vdim:(head + 1) * vdim]
            if kind == "delta":
                run = lambda f: plain.delta_rule(unit(q[f:, group]) * dim ** -0.5, unit(k[f:, group]), v[f:],
                                                 plain.sigmoid(s["b"][f:, head]), decay[f:, head])
            else:
                run = lambda f: plain.dual_scan(v[f:], k[f:, group], q[f:, group], step[f:, head], decay[f:, head], skip[head])
            want, last = run(0)
            have = np.concatenate(got[row])[:, head * vdim:(head + 1) * vdim]
            assert np.abs(have - want).max() < 2e-4 * max(1.0, np.abs(want).max()), (row, head)
            assert np.abs(state[slots[row], head].double().cpu().numpy().T - last).max() < 2e-4 * max(1.0, np.abs(last).max())
            if total > 30 and dim > 1:       # without the first token's write the last output is another
                again, _ = run(1)
                close = 2e-4 * max(1.0, np.abs(want[-1]).max())
                assert np.abs(have[-1] - want[-1]).max() < close and np.abs(again[-1] - want[-1]).max() > 10 * close


@gpu
@pytest.mark.parametrize("dtype, head_dim, heads, kv_heads, context, page, rows, far", [
    (torch.bfloat16, 64, 8, 2, 700, 16, 16, 150), (torch.bfloat16, 128, 4, 4, 2300, 16, 32, 1900),
    (torch.bfloat16, 128, 2, 1, 300, 16, 6, 40000), (torch.bfloat16, 64, 6, 6, 1500, 32, 8, 20), (torch.float32, 64, 4, 2, 500, 8, 12, 129),
    (torch.float32, 24, 3, 1, 200, 4, 7, 31), (torch.bfloat16, 40, 6, 3, 300, 8, 10, 64), (torch.bfloat16, 64, 4, 2, 400, 4, 9, 200)])
def test_a_bias_per_head_and_distance_in_every_attention_kernel(dtype, head_dim, heads, kv_heads, context, page, rows, far):
    """Scores get a number by head and distance in the general kernel, the
    split-key decode kernels and both tensor-core prompt kernels, with tables
    that end inside a key tile, reach over many, or are too long for shared
    memory. A few distances carry a large number (1, the last of the near half,
    one on either side of the table's far end), so that a distance off by one
    would show; one query looks far back and one at a page's first row."""
    from metallix_b200 import ops
    from metallix_b200.parts.attention import distance_rows
    rng = np.random.default_rng(head_dim + context)
    scale, tail = 0.15, 24
    spread = np.asarray(distance_rows(rows, far))
    table = rng.normal(size=(rows, heads))
    table[1] += np.log(context) - 1.0
    table[rows // 2 - 1] += np.log(context) - 1.0
    if far < context:
        table[rows - 2] += 4.0
    by_distance = rounded(np.ascontiguousarray(table[spread].T), torch.float32)            # [heads, distances]
    keys = rng.normal(size=(context, kv_heads, head_dim)) * 0.5
    values = rng.normal(size=(context, kv_heads, head_dim))
    q = rng.normal(size=(tail, heads, head_dim)) * 0.5
    group, first = heads // kv_heads, context - tail

    def look_for(t, key, factor=6.0):
        keys[key] *= factor
        q[t] = np.repeat(keys[key], group, axis=0) * 1.5

    look_for(tail - 1, 5)                      # far back
    look_for(10, (first + 10) // page * page)      # a page's first row
    keys, values, q = rounded(keys, dtype), rounded(values, dtype), rounded(q, dtype)
    pages = -(-context // page)
    order = rng.permutation(pages + 2)[:pages]
    pool = torch.zeros((pages + 2, 2, kv_heads, page, head_dim), dtype=dtype, device="cuda")
    for p in range(pages):
        span = slice(p * page, min((p + 1) * page, context))
        n = span.stop - span.start
        pool[order[p], 0, :, :n] = dev(keys[span].transpose(1, 0, 2), dtype)
        pool[order[p], 1, :, :n] = dev(values[span].transpose(1, 0, 2), dtype)
    positions = np.arange(first, context)
    k_all, v_all = np.repeat(keys, group, axis=1), np.repeat(values, group, axis=1)

    def attended(numbers):
        out = np.zeros((tail, heads, head_dim))
        for t, p in enumerate(positions):
            s = np.einsum("hd,jhd->hj", q[t], k_all[:p + 1]) * scale
            s = s + numbers[:, np.minimum(p - np.arange(p + 1), numbers.shape[1] - 1)]
            out[t] = np.einsum("hj,jhd->hd", plain.softmax(s, np.ones_like(s, dtype=bool)), v_all[:p + 1])
        return out

    want = attended(by_distance)
    tolerance = 3e-5 if dtype == torch.float32 else 3e-2
    assert np.abs(want - attended(np.zeros((heads, 1)))).max() > 10 * tolerance       # the numbers show
    assert np.abs(want - attended(by_distance[:, 1:])).max() > 5 * tolerance          # ... and a distance off by one
    tables, bias = dev(order[None, :], torch.int32), dev(by_distance)
    out = torch.empty((tail, heads, head_dim), dtype=dtype, device="cuda")
    ops.paged_attention_tile(dev(q, dtype), pool, out, tables, dev([0, 0], torch.int32), dev([0, 16], torch.int32),
                             dev([16, tail - 16], torch.int32), dev(positions, torch.int32), scale, bias=bias)
    ops.check_status("cuda")
    assert np.abs(out.double().cpu().numpy() - want).max() < tolerance
    if ops.decode_attention_supported(head_dim, heads, kv_heads, dtype):
        for t in (0, 7, 10, tail - 1):      # each as a single decoded token behind its context
            for resident in (444, 0):       # blocks that walk over tiles, and a block per tile
                ops.set_decode_resident_blocks(resident)
                one = torch.empty((1, heads, head_dim), dtype=dtype, device="cuda")
                ops.paged_attention_decode(dev(q[t:t + 1], dtype), pool, one, tables, dev([0], torch.int32), dev([0], torch.int32),
                                           dev(positions[t:t + 1], torch.int32), scale, int(positions[t]) + 1, bias=bias)
                ops.check_status("cuda")
                assert np.abs(one.double().cpu().numpy()[0] - want[t]).max() < tolerance, (t, resident)
            ops.set_decode_resident_blocks(444)
    if ops.flash_prefill_supported(head_dim, heads, kv_heads, dtype):
        for kernel in ("tcgen05", "mma"):
            if kernel == "tcgen05" and not ops.flash_prefill_tcgen05_supported(head_dim, heads, kv_heads, page, dtype):
                continue
            for longest in (0, context):
                out.zero_()
                ops.flash_prefill(dev(q, dtype), pool, out, tables, dev([0], torch.int32), dev([0], torch.int32),
                                  dev([tail], torch.int32), dev(positions, torch.int32), scale, kernel=kernel,
                                  longest_context=longest, bias=bias)
                ops.check_status("cuda")
                assert np.abs(out.double().cpu().numpy() - want).max() < tolerance, (kernel, longest)


@gpu
@pytest.mark.parametrize("head_dim", [64, 128])
def test_a_decode_step_of_many_rows_walks_tiles_with_its_biases(head_dim):
    """Many rows with long contexts: every block of the resident kernel walks
    over several key tiles, each with biases of its own distances; and the
    same step joined with the output projection."""
    from metallix_b200 import ops
    rng = np.random.default_rng(3)
    rows, heads, kv_heads, context, page, scale = 3, 4, 2, 3000, 16, 0.12
    by_distance = rounded(rng.normal(size=(heads, 1500)) * 1.5, torch.float32)
    pages = -(-context // page)
    keys, values = (rounded(rng.normal(size=(context, kv_heads, head_dim)), torch.bfloat16) for _ in range(2))
    pool = torch.zeros((pages, 2, kv_heads, page, head_dim), dtype=torch.bfloat16, device="cuda")
    padded = lambda x: np.concatenate([x, np.zeros((pages * page - context,) + x.shape[1:])])
    for plane, x in enumerate((keys, values)):
        pool[:, plane] = dev(padded(x).reshape(pages, page, kv_heads, head_dim).transpose(0, 2, 1, 3), torch.bfloat16)
    positions = np.asarray([context - 1, 1700, 90])
    q = rounded(rng.normal(size=(rows, heads, head_dim)), torch.bfloat16)
    want = np.zeros((rows, heads, head_dim))
    for t, p in enumerate(positions):
        s = np.einsum("hd,jhd->hj", q[t], np.repeat(keys[:p + 1], 2, axis=1)) * scale
        s = s + by_distance[:, np.minimum(p - np.arange(p + 1), 1499)]
        want[t] = np.einsum("hj,jhd->hd", plain.softmax(s, np.ones_like(s, dtype=bool)), np.repeat(values[:p + 1], 2, axis=1))
    table = torch.arange(pages, dtype=torch.int32, device="cuda").repeat(rows, 1)
    index = torch.arange(rows, dtype=torch.int32, device="cuda")
    try:
        for resident in (12, 444, 0):
            ops.set_decode_resident_blocks(resident)
            out = torch.empty((rows, heads, head_dim), dtype=torch.bfloat16, device="cuda")
            ops.paged_attention_decode(dev(q, torch.bfloat16), pool, out, table, index, index, dev(positions, torch.int32), scale,
                                       context, bias=dev(by_distance))
            ops.check_status("cuda")
            assert np.abs(out.double().cpu().numpy() - want).max() < 3e-2, resident
            w = rounded(rng.normal(size=(256, heads * head_dim)) * 0.1, torch.bfloat16)
            parts = ops.paged_attention_decode_project(dev(q, torch.bfloat16), pool, table, index, index, dev(positions, torch.int32),
                                                       scale, context, dev(w, torch.bfloat16), bias=dev(by_distance))
            ops.check_status("cuda")
            assert np.abs(parts.sum(0).double().cpu().numpy() - want.reshape(rows, -1) @ w.T).max() < 5e-2
    finally:
        ops.set_decode_resident_blocks(444)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("head_dim, heads, kv_heads, scope, normed", [(64, 4, 2, "head", True), (128, 2, 2, "head", False),
                                                                      (18, 3, 1, "head", True), (24, 2, 1, "projection", True)])
def test_query_factors_beside_norms_and_the_cache_write(dtype, head_dim, heads, kv_heads, scope, normed):
    """Queries times a factor of their position, in the three kernels that
    write them; keys and values are not touched by it, and the values are the
    keys as projected."""
    from metallix_b200 import ops
    from metallix_b200.config.spec import PartSpec
    from metallix_b200.parts.registry import Runtime, WeightStore, build_part
    rng = np.random.default_rng(head_dim)
    positions, eps, page = [0, 4, 5, 9, 39, 6], 1e-5, 8
    tokens = len(positions)
    part = build_part("position", PartSpec("log_temperature", {"coef": 0.7, "every": 5}), WeightStore({}),
                      Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=40))
    q, k = rounded(rng.normal(size=(tokens, heads * head_dim)), dtype), rounded(rng.normal(size=(tokens, kv_heads * head_dim)), dtype)
    width = lambda n: head_dim if scope == "head" else n * head_dim
    wq, wk = (rounded(1.0 + rng.normal(size=width(n)) * 0.2, torch.float32) if normed else None for n in (heads, kv_heads))

    def over(x, w, n):
        if w is None:
            return x.reshape(tokens, n, head_dim)
        if scope == "head":
            return plain.over_rms(x.reshape(tokens, n, head_dim), eps) * w
        return (plain.over_rms(x, eps) * w).reshape(tokens, n, head_dim)

    factors = plain.query_temperature(40, {"coef": 0.7, "every": 5})[positions]
    q_out = torch.empty((tokens, heads, head_dim), dtype=dtype, device="cuda")
    pool = torch.zeros((2, 2, kv_heads, page, head_dim), dtype=dtype, device="cuda")
    slots = [3, 8, 15, -1, 0, 9]
    both = dev(np.concatenate([q, k], axis=1), dtype)
    keys = both[:, heads * head_dim:]
    ops.qk_norm_rope_cache(both[:, :heads * head_dim], keys, keys, q_out, pool, dev(slots, torch.int32), dev(positions, torch.int32),
                           dev(wq) if normed else None, dev(wk) if normed else None, None, None, eps, norm_scope=scope,
                           q_factors=part.factors)
    ops.check_status("cuda")
    tolerance = 2e-5 if dtype == torch.float32 else 4e-2
    assert np.abs(q_out.double().cpu().numpy() - over(q, wq, heads) * factors[:, None, None]).max() < tolerance
    want_k = over(k, wk, kv_heads)
    for t, slot in enumerate(slots):
        if slot >= 0:
            row = pool[slot // page, :, :, slot % page].double().cpu().numpy()
            assert np.abs(row[0] - want_k[t]).max() < tolerance
            assert np.array_equal(row[1], k[t].reshape(kv_heads, head_dim))
    assert float(pool[1, :, :, 6].abs().max()) == 0.0
    alone = ops.norm_rotate_heads(both[:, :heads * head_dim], head_dim, dev(positions, torch.int32), factors=part.factors)
    assert np.abs(alone.double().cpu().numpy() - q.reshape(tokens, heads, head_dim) * factors[:, None, None]).max() < tolerance


@gpu
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("size", [72, 128, 2056, 8192])
def test_two_outputs_behind_norms_of_their_own_and_the_next_norm(out_dtype, size):
    """x += a norm(left + bias) + b norm(right), then the next norm of x, with
    either type on either side, left in summands, without the next norm."""
    from metallix_b200 import ops
    rng = np.random.default_rng(size)
    rows, eps = 5, (1e-5, 1e-3, 1e-6)
    x = rounded(rng.normal(size=(rows, size)) * 2.0, torch.float32)
    wl, wr, w = (rounded(1.0 + rng.normal(size=size) * 0.2, torch.float32) for _ in range(3))
    bias = rounded(rng.normal(size=size), torch.float32)
    tolerance = 2e-5 if out_dtype == torch.float32 else 4e-2
    for left_type, right_type, biased, parts in ((torch.bfloat16, torch.float32, True, 1), (torch.float32, torch.bfloat16, False, 1),
                                                 (torch.float32, torch.bfloat16, True, 3), (torch.bfloat16, torch.bfloat16, True, 1)):
        left = rounded(rng.normal(size=(parts, rows, size)) * 0.3, left_type)
        right = rounded(rng.normal(size=(rows, size)) * 5.0, right_type)
        total = x + 0.5 * plain.over_rms(left.sum(0) + (bias if biased else 0.0), eps[0]) * wl - 0.25 * plain.over_rms(right, eps[1]) * wr
        stream = dev(x)
        given = dev(left if parts > 1 else left[0], left_type)
        got = ops.pair_norm(stream, given, dev(right, right_type), dev(wl), dev(wr), eps[0], eps[1], 0.5, -0.25,
                            left_bias=dev(bias) if biased else None, weight=dev(w), eps=eps[2], out_dtype=out_dtype)
        assert np.abs(stream.double().cpu().numpy() - total).max() < 2e-5
        assert np.abs(got.double().cpu().numpy() - plain.over_rms(total, eps[2]) * w).max() < tolerance
        stream = dev(x)
        assert ops.pair_norm(stream, given, dev(right, right_type), dev(wl), dev(wr), eps[0], eps[1], 0.5, -0.25,
                             left_bias=dev(bias) if biased else None) is None
        assert np.abs(stream.double().cpu().numpy() - total).max() < 2e-5


@gpu
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("parts, part_size", [(1, 60), (3, 20), (4, 7), (1, 9000), (2, 512)])
def test_a_gate_ahead_of_a_norm_in_parts_and_one_behind_a_heads_norm(out_dtype, parts, part_size):
    from metallix_b200 import ops
    rng = np.random.default_rng(part_size)
    tokens, width, eps = 6, parts * part_size, 1e-4
    x = rounded(rng.normal(size=(tokens, width)) * 0.1, torch.float32)
    w = rounded(1.0 + rng.normal(size=width) * 0.3, torch.float32)
    tolerance = 3e-5 if out_dtype == torch.float32 else 8e-3      # of the largest value
    for gate_type in (torch.float32, torch.bfloat16):
        gate = rounded(rng.normal(size=(tokens, width)) * 2.0, gate_type)
        wide = dev(np.concatenate([np.zeros((tokens, 3)), gate, np.zeros((tokens, 5))], axis=1), gate_type)[:, 3:3 + width]
        for name, act in (("silu", plain.silu), ("sigmoid", plain.sigmoid)):
            got = ops.gated_norm(dev(x), dev(w), wide, parts, eps, out_dtype, activation=name)
            want = plain.over_rms((x * act(gate)).reshape(tokens, parts, part_size), eps).reshape(tokens, width) * w
            assert np.abs(got.double().cpu().numpy() - want).max() < tolerance * np.abs(want).max(), name
            got = ops.head_norm_gate(dev(x), dev(w), wide, parts, eps, out_dtype, activation=name)
            want = plain.over_rms(x.reshape(tokens, parts, part_size), eps).reshape(tokens, width) * w * act(gate)
            assert np.abs(got.double().cpu().numpy() - want).max() < tolerance * np.abs(want).max(), name


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_join_ahead_of_a_pass(dtype):
    """[x + pending | x0] in the compute type, through the part with each kind
    of thing that may be pending, and the pass's vector joining every row in
    the next norm's kernel or alone."""
    from metallix_b200 import ops
    from metallix_b200.config.spec import PartSpec
    from metallix_b200.parts.norm import RMSNorm
    from metallix_b200.parts.parallel import NormedPair
    from metallix_b200.parts.registry import Runtime, WeightStore, build_part, settle
    rng = np.random.default_rng(5)
    tokens, size, turns = 7, 72, 3
    runtime = Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=16)
    weight = rounded(rng.normal(size=(size, 2 * size)) * 0.1, torch.bfloat16)
    steps = rounded(rng.normal(size=(turns, size)), torch.bfloat16)
    part = build_part("join", PartSpec("mix_first", {"hidden_size": size, "weight": "w", "steps": "s", "turns": turns}),
                      WeightStore({"w": torch.tensor(weight), "s": torch.tensor(steps)}), runtime)
    x, x0 = (rounded(rng.normal(size=(tokens, size)), torch.float32) for _ in range(2))
    tolerance = 1e-5 if dtype == torch.float32 else 3e-2
    ones = RMSNorm(torch.ones(size), 1e-5, runtime)
    for kind in ("none", "float32", "bfloat16", "pair", "row"):
        delta = rounded(rng.normal(size=(tokens, size)), torch.bfloat16 if kind == "bfloat16" else torch.float32)
        other = rounded(rng.normal(size=(tokens, size)), torch.float32)
        pending, added = None, 0.0
        if kind in ("float32", "bfloat16"):
            pending, added = dev(delta, getattr(torch, kind)), delta
        elif kind == "pair":
            pending = NormedPair(dev(delta), dev(other), ones, ones, (0.5, 0.5))
            added = 0.5 * plain.over_rms(delta, 1e-5) + 0.5 * plain.over_rms(other, 1e-5)
        elif kind == "row":
            pending, added = dev(delta[0]), delta[0]
        mixed, left = part.forward(dev(x), pending, dev(x0), 2)
        want = np.concatenate([x + added, x0], axis=1) @ weight.T
        assert mixed.dtype == torch.float32 and np.abs(mixed.double().cpu().numpy() - want).max() < tolerance * 3
        have = mixed.double().cpu().numpy() + steps[2]
        alone = mixed.clone()
        settle(alone, left)
        assert np.abs(alone.double().cpu().numpy() - have).max() < 1e-5
        normed = ones.add_forward(mixed, left, torch.float32)
        assert np.abs(mixed.double().cpu().numpy() - have).max() < 1e-5
        assert np.abs(normed.double().cpu().numpy() - plain.over_rms(have, 1e-5)).max() < 1e-5
    for odd in (7, 70):      # rows that the vector form does not take
        stream, row = rounded(rng.normal(size=(4, odd)), torch.float32), rounded(rng.normal(size=odd), torch.float32)
        got = dev(stream)
        normed = ops.add_rmsnorm(got, dev(row), torch.ones(odd, device="cuda"), 1e-5, torch.float32)
        assert np.abs(normed.double().cpu().numpy() - plain.over_rms(stream + row, 1e-5)).max() < 1e-5


@gpu
@pytest.mark.parametrize("experts, top", [(6, 2), (8, 1), (3, 3), (1, 1), (64, 6), (300, 5)])
def test_router_that_weighs_the_chosen_alone(experts, top):
    """The largest logits, bias included, are chosen; their weights are the
    softmax over the chosen. Logits are large enough that a softmax over all
    of them would leave the chosen ones of some rows nothing."""
    from metallix_b200 import ops
    rng = np.random.default_rng(experts * top)
    tokens = 37
    logits = rounded(rng.normal(size=(tokens, experts)) * 30.0, torch.float32)
    bias = rounded(rng.normal(size=experts) * 20.0, torch.float32)
    wide = dev(np.concatenate([logits, np.zeros((tokens, 3))], axis=1))
    chosen, weights, dense_weights, on_identity = ops.route_experts(wide[:, :experts], dev(bias), experts, top, scores="chosen")
    want_chosen, want_weights = plain.choose_experts(logits + bias, top)
    assert np.array_equal(chosen.cpu().numpy(), want_chosen)
    assert np.abs(weights.double().cpu().numpy() - want_weights).max() < 1e-4
    assert float(on_identity.abs().max()) == 0.0 and np.abs(dense_weights.sum(dim=1).double().cpu().numpy() - 1.0).max() < 1e-4


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, shared", [(1, 24), (5, 40), (300, 40), (5, 0)])
def test_experts_with_a_shared_one_that_has_no_gate(dtype, tokens, shared):
    """Experts of squared relu through the part itself, row by row and
    grouped, with a shared expert as wide as the others or not."""
    from metallix_b200.config.kokolorn import ChosenExperts
    from metallix_b200.parts.registry import Runtime, WeightStore, build_part
    rng = np.random.default_rng(tokens + shared)
    hidden, ff, experts, top = 64, 40, 5, 2
    typed = ChosenExperts(ff=ff, experts=experts, top=top, shared_ff=shared)
    tensors = {k: rounded(rng.normal(size=shape) * 0.3, torch.bfloat16) for k, shape in typed.shapes("m", hidden).items()}
    part = build_part("feed_forward", typed.part("m", hidden), WeightStore({k: torch.tensor(v) for k, v in tensors.items()}),
                      Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=16))
    h = rounded(rng.normal(size=(tokens, hidden)), dtype)
    got = part.forward(dev(h, dtype), None).double().cpu().numpy()
    want = plain.expert_mixture(h, tensors, "m", typed.to_dict())
    errors = np.abs(got - want).max(axis=1)
    if dtype == torch.float32:
        assert errors.max() < 1e-4 * max(1.0, np.abs(want).max())
    else:       # a close call of the router may go the other way for a token in a hundred
        assert np.quantile(errors, 0.97) < 3e-2 * max(1.0, np.abs(want).max())


@gpu
@pytest.mark.parametrize("rows", [1, 8, 40, 1600])
def test_gated_feed_forward_with_clamped_halves(rows):
    """Both halves bounded, in every kernel that holds the activation: the
    pass of its own, the few-row products' epilogue, the tensor-core product's.
    The products reach well beyond the limit on both sides."""
    from metallix_b200 import ops, tensor_core
    rng = np.random.default_rng(rows)
    hidden, ff, limit = 128, 192, 1.25
    x = rounded(rng.normal(size=(rows, hidden)), torch.bfloat16)
    w = rounded(rng.normal(size=(2 * ff, hidden)) * 0.2, torch.bfloat16)
    gate_up = rounded(x @ w.T, torch.bfloat16)
    g, u = np.minimum(gate_up[:, :ff], limit), np.clip(gate_up[:, ff:], -limit, limit)
    want = g * plain.sigmoid(1.702 * g) * (u + 1.0)
    assert (gate_up > limit).mean() > 0.1 and (gate_up < -limit).mean() > 0.1
    tolerance = 3e-2 * max(1.0, np.abs(want).max())
    for dtype in (torch.float32, torch.bfloat16):
        got = ops.silu_mul(dev(rounded(gate_up, dtype), dtype), activation="clamped", limit=limit)
        assert np.abs(got.double().cpu().numpy() - want).max() < (1e-5 if dtype == torch.float32 else tolerance)
    if rows <= 16:
        for kernel in ("stream", "load"):
            got = ops.gemm_skinny(dev(x, torch.bfloat16), dev(w, torch.bfloat16), swiglu=True, kernel=kernel, activation="clamped",
                                  limit=limit)
            assert np.abs(got.double().cpu().numpy() - want).max() < tolerance, kernel
    got = tensor_core.gemm_swiglu(dev(x, torch.bfloat16), dev(w, torch.bfloat16), activation="clamped", limit=limit)
    assert np.abs(got.double().cpu().numpy() - want).max() < tolerance
    far = dev(np.asarray([[-300.0, 500.0, 2.0, -700.0]]))      # gates far outside: 0 and the limit's own value
    got = ops.silu_mul(far, activation="clamped", limit=limit)[0].double().cpu().numpy()
    assert abs(got[0]) < 1e-6 and np.isclose(got[1], limit * plain.sigmoid(1.702 * limit) * (1.0 - limit))


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_side_by_side_mixers_as_a_plain_result_and_as_a_pending_one(folders, dtype):
    """The pair through ``forward`` (a tensor) is what the pending form adds."""
    from metallix_b200.parts.registry import CacheView, StepContext
    name = "small"
    engine = make_engine(folders, name, dtype)
    _, config, tensors, _ = folders[name]
    mixer = engine.model.blocks[1].mixer
    h = np.random.default_rng(1).normal(size=(11, 72))
    rounded_h = rounded(h, engine.dtype)
    ints = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")

    def view():
        members = []
        for need in mixer.cache_need().members:
            if need.kind == "kv_pages":
                pool = torch.zeros((2, 2, need.kv_heads, 8, need.head_dim), dtype=engine.dtype, device="cuda")
                members.append(CacheView(need, pool=pool, block_tables=ints([[0, 1]]), slots=ints(range(11))))
            else:
                members.append(CacheView(need, members=[
                    CacheView(n, state=torch.zeros((1,) + tuple(n.state_shape), device="cuda")) for n in need.members]))
        return CacheView(mixer.cache_need(), members=members)

    def context():
        return StepContext(device=torch.device("cuda"), dtype=engine.dtype, num_tokens=11, num_requests=1, positions=ints(range(11)),
                           token_request=ints([0] * 11), request_slots=ints([0]), request_offsets=[0, 11], request_positions=[0])

    want = plain.side_by_side(rounded_h, {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}, "l1.mix",
                              config["layers"][1]["mixer"], config["norm"]["eps"])
    x = dev(rounded_h, engine.dtype)
    whole = mixer.forward(x, context(), view())
    stream = torch.zeros((11, 72), device="cuda")
    mixer.forward_pending(x, context(), view()).settle(stream)
    engine.check()
    tolerance = 1e-4 if dtype == "float32" else 8e-2
    assert torch.equal(whole, stream) and np.abs(whole.double().cpu().numpy() - want).max() < tolerance
    left = mixer.left.forward(x, context(), view().members[0]).double().cpu().numpy()      # alone, its output bias included
    want = plain.keys_as_values_attention(rounded_h, {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()},
                                          "l1.mix.left", config["layers"][1]["mixer"]["left"], 1e-6, norms=False, biased_output=True)
    assert np.abs(left - want).max() < tolerance


# ------------------------------------------------- the engine: whole prompts
@gpu
@pytest.mark.parametrize("name, dtype", CASES)
def test_whole_prompts_layer_by_layer(folders, name, dtype):
    """A prompt in one step: the residual stream after every layer run, then
    the logits at every position; a single token; two tokens."""
    from metallix_b200.engine import StepEntry
    engine = make_engine(folders, name, dtype)
    _, config, tensors, _ = folders[name]
    ids = random_ids(7, 45, config["vocab"])
    want_taps = []
    want = plain.forward_logits(config, tensors, ids, want_taps)
    got_taps = []
    logits = engine.step([StepEntry("a", ids, list(range(len(ids))))], tap=lambda i, r: got_taps.append(r.double().cpu().numpy()))
    engine.check()
    assert len(got_taps) == len(want_taps) == len(plain.layer_runs(config))
    for index, (have, should) in enumerate(zip(got_taps, want_taps)):
        errors = np.abs(have - should).max(axis=1) / max(1.0, np.abs(should).max())
        if dtype == "float32":
            assert errors.max() < bound(name, dtype), index
        else:       # a router's close call may send a token or two to another expert
            assert np.quantile(errors, 0.9) < 2 * bound(name, dtype), index
    if dtype == "float32":
        assert np.abs(logits.double().cpu().numpy() - want).max() < bound(name, dtype)
    else:
        compare_replay(name, dtype, {("a", t): row for t, row in enumerate(logits.double().cpu().numpy())}, {"a": want})
    engine.release("a")
    for length in (1, 2):
        logits = engine.step([StepEntry("b", ids[:length], list(range(length)))])
        assert np.abs(logits.double().cpu().numpy() - want[:length]).max() < (bound(name, dtype) if dtype == "float32" else 1.5)
        engine.release("b")
    engine.check()


@gpu
@pytest.mark.parametrize("name, dtype", CASES)
def test_decoding_and_portions_against_whole_prompts(folders, name, dtype):
    """The same requests as whole prompts, with their tails decoded one by one
    (over more tokens than the small tables' far ends), and in portions of
    changing size down to two tokens (and one)."""
    from metallix_b200.engine import StepEntry
    requests = some_requests(name, 40, (75, 9, 33, 400 if name == "wide" else 50))
    reference = reference_logits(folders, name, requests)
    for schedule in (cuts.whole(requests), cuts.tail_by_one(requests, tail=45), cuts.ragged(requests),
                     cuts.ragged(requests, sizes=(2, 2, 3, 1, 2, 4, 9, 2))):
        engine = make_engine(folders, name, dtype, pages=64, max_requests=2)
        _, seen = cuts.replay(engine, schedule, reference, StepEntry)
        compare_replay(name, dtype, seen, reference)


@gpu
@pytest.mark.parametrize("name, dtype", CASES)
def test_mixed_batches_with_pages_and_slots_that_come_back(folders, name, dtype):
    """Up to four requests live at once in a pool made for just that many:
    portions beside single tokens, requests that sit a step out, ended requests
    whose pages and state slots the next ones take over. Each position's
    logits equal those of the request run alone."""
    from metallix_b200.engine import StepEntry
    requests = some_requests(name, 60, (70, 41, 5, 90, 23, 1, 37, 64, 2, 55))
    reference = reference_logits(folders, name, requests)
    steps, peak = cuts.mixed(requests, seed=5, max_live=4)
    page = folders[name][3]
    engine = make_engine(folders, name, dtype, pages=-(-peak // page), max_requests=4)
    _, mixed_seen = cuts.replay(engine, steps, reference, StepEntry)
    compare_replay(name, dtype, mixed_seen, reference)
    assert engine.manager.pages_reused() > 0 and len(requests) > engine.manager.max_requests()
    if dtype == "float32":     # against the engine itself, each request alone: rounding of the products only
        alone = make_engine(folders, name, dtype, pages=48, max_requests=2)
        _, alone_seen = cuts.replay(alone, cuts.whole(requests), reference, StepEntry)
        gap = max(float(np.abs(row - alone_seen[key]).max()) for key, row in mixed_seen.items())
        assert gap < 0.3 * bound(name, dtype)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_that_decides_the_output(folders, dtype):
    """Attention through the engine's cache where one early token decides what
    a late one answers: the projections of one layer are made so that the last
    token's query is the early token's key (at a page's border or the
    sequence's start) and nobody else's, in a prompt and decoded alone; with
    another token at that early place the logits are far away."""
    from metallix_b200.config import KokolornConfig
    from metallix_b200.engine import Engine, StepEntry
    rng = np.random.default_rng(12)
    raw = {"architecture": "Kokolorn", "vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
           "layers": [layer("attention", attention(2, 1, 64, 0.5, (0.1, 40)), None)]}
    tensors = random_model(raw, 4)
    tensors["embed"] = rng.normal(size=(64, 64))
    tensors["embed"][62] = np.roll(tensors["embed"][63], 1)
    tensors["l0.mix.q"] = np.concatenate([np.roll(np.eye(64), 1, axis=0)] * 2)      # q of 63 = k of 62
    tensors["l0.mix.k"] = np.eye(64)
    tensors["l0.mix.o"] = np.concatenate([np.eye(64), np.zeros((64, 64))], axis=1)
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.norm1", "final.norm"):
        tensors[name] = tensors[name] * 0.0
    for name in ("l0.mix.q.norm", "l0.mix.k.norm"):
        tensors[name] = np.ones(64)
    tensors = {name: rounded(value, torch.bfloat16) for name, value in tensors.items()}
    for early in (0, 15, 16, 31, 130):
        ids = [int(t) for t in rng.integers(1, 60, size=200)]
        ids[early] = 62
        ids.append(63)
        want = plain.forward_logits(raw, tensors, ids)[-1]
        other = plain.forward_logits(raw, tensors, ids[:early] + [7] + ids[early + 1:])[-1]
        tolerance = 1e-4 if dtype == "float32" else 1.5e-1
        assert np.abs(want - other).max() > 8 * tolerance
        for split in (len(ids), len(ids) - 1):
            engine = Engine(KokolornConfig.from_dict(raw), {k: torch.tensor(v, dtype=torch.float32) for k, v in tensors.items()},
                            dtype=dtype, page_tokens=16, num_pages=16, max_requests=1)
            logits = None
            for part in (ids[:split], ids[split:]):
                if part:
                    logits = engine.step([StepEntry("a", part, [len(part) - 1])])
            engine.check()
            assert np.abs(logits[0].double().cpu().numpy() - want).max() < tolerance, (early, split)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_captured_steps(folders, dtype):
    """Three requests decoded together for 160 steps (captured graphs), one of
    them leaving on the way and another joining with a prompt: the recurrent
    states of every pass, the convolutions' inputs and the pages stay each
    request's own."""
    from metallix_b200.engine import StepEntry
    name = "small"
    requests = some_requests(name, 80, (190, 170, 120))
    reference = reference_logits(folders, name, requests)
    engine = make_engine(folders, name, dtype, pages=80, max_requests=3)
    heads = {"r0": 30, "r1": 12}
    seen = {}
    engine.step([StepEntry(k, requests[k][:n], [n - 1]) for k, n in heads.items()])
    at = dict(heads)
    for step in range(160):
        if step == 40:       # r2 joins with a prompt of its own beside the decoded tokens
            at["r2"] = 0
        entries, places = [], []
        for key in list(at):
            ids = requests[key]
            if at[key] >= len(ids):
                engine.release(key)
                del at[key]
                continue
            count = 17 if key == "r2" and at[key] == 0 else 1
            entries.append(StepEntry(key, ids[at[key]:at[key] + count], [count - 1]))
            places.append((key, at[key] + count - 1))
            at[key] += count
        if not entries:
            break
        logits = engine.step(entries).double().cpu().numpy()
        for row, place in enumerate(places):
            seen[place] = logits[row]
    engine.check()
    assert len(seen) > 400
    compare_replay(name, dtype, seen, reference)
    assert engine.graphs is not None and engine.graphs.sizes_captured()      # decode steps did run as graphs


@gpu
def test_fork_copies_pages_and_state(folders):
    from metallix_b200.engine import StepEntry
    name = "small"
    _, config, tensors, _ = folders[name]
    ids = random_ids(3, 40, config["vocab"])
    other = ids[:22] + random_ids(4, 18, config["vocab"])
    engine = make_engine(folders, name, "float32", pages=64)
    engine.step([StepEntry("p", ids[:22], [])])
    engine.fork("p", "c")
    a = engine.step([StepEntry("p", ids[22:], list(range(18))), StepEntry("c", other[22:], list(range(18)))])
    engine.check()
    want = np.concatenate([plain.forward_logits(config, tensors, ids)[22:], plain.forward_logits(config, tensors, other)[22:]])
    assert np.abs(a.double().cpu().numpy() - want).max() < TOL["float32"]


# ------------------------------------- generation, scheduler, command line
@gpu
@pytest.mark.parametrize("name, dtype", [("small", "float32"), ("small", "bfloat16"), ("wide", "bfloat16"), ("bare", "float32")])
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    """``generate`` (scheduler, continuous batching, captured decode steps):
    every generated token is the plain side's argmax, or (bfloat16) within a
    near tie of it."""
    from metallix_b200.engine.generate import generate
    _, config, tensors, _ = folders[name]
    engine = make_engine(folders, name, dtype, pages=64, max_requests=4)
    prompts = [random_ids(90 + n, length, config["vocab"]) for n, length in enumerate((5, 31, 1, 12, 18, 2))]
    results = generate(engine, prompts, max_new_tokens=12, eos_ids=())
    for prompt, result in zip(prompts, results):
        assert len(result.generated_ids) == 12 and not result.failed
        ids = list(prompt)
        for token in result.generated_ids:
            row = plain.forward_logits(config, tensors, ids)[-1]
            best = int(np.argmax(row))
            if token != best:
                assert dtype == "bfloat16" and row[best] - row[token] < 0.5, (dtype, token, best)
            ids.append(token)


@gpu
def test_trace_program_and_command_line(folders, tmp_path):
    """bin/trace_run on a mixed schedule and bin/mxb gen, as programs."""
    name = "small"
    folder, config, tensors, page = folders[name]
    requests = some_requests(name, 70, (30, 12, 44))
    reference = reference_logits(folders, name, requests)
    steps, peak = cuts.mixed(requests, seed=9, max_live=2, decode_tail=6)
    out = tmp_path / "logits"
    done = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                           "--out", str(out), "--max-tokens", str(peak)],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done ")] == [f"done {s['step']}" for s in steps]
    offsets = {}
    for step in steps:
        for e in step["entries"]:
            offsets.setdefault(e["id"], 0)
        want = cuts.expected_rows(step, offsets, reference)
        if want is not None:
            got = np.fromfile(out / f"{step['step']}.f32", dtype="<f4").reshape(want.shape)
            assert np.abs(got - want).max() < TOL["float32"]
        for e in step["entries"]:
            offsets[e["id"]] += len(e["tokens"])
    prompt = requests["r1"]
    done = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "mxb"), "gen", "--model", folder, "--input-ids",
                           ",".join(map(str, prompt)), "--max-tokens", "4", "--dtype", "float32", "--verify-cache"],
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    receipt = json.loads(done.stdout.strip().splitlines()[-1])
    ids = list(prompt)
    for _ in range(4):
        ids.append(int(np.argmax(plain.forward_logits(config, tensors, ids)[-1])))
    assert receipt["generated_ids"] == ids[len(prompt):]
    assert receipt["cache_comparisons"]["logits_within_bound"]
