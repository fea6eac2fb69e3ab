"""The Mekuvik decoder in the engine against the plain implementation
(``plain_mekuvik.py``): its configuration and mechanisms one at a time, then
whole prompts layer run by layer run, decoding through the cache and the state,
portions, mixed batches, pages and slots that come back, keys far back, at page
borders, on either side of a window's edge and of the last kept position, the
first tokens, long decoding, generation through the scheduler and the trace
program. Every model here is tiny, made for the test with random weights, and
differs from layer to layer."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_mekuvik as plain
import replay_helpers as cuts
from conftest import ROOT, random_ids


# ------------------------------------------------------------ configurations
def lightning(heads, dim, vdim, decay):
    out = {"heads": heads, "dim": dim, "decay": decay}
    if vdim:
        out["vdim"] = vdim
    return out


def attention(heads, kv_heads, dim, vdim, scale, rot=None, mask=None):
    out = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads:
        out["kv_heads"] = kv_heads
    if vdim:
        out["vdim"] = vdim
    if rot:
        out["rot"] = {"base": rot[0], "dims": rot[1]}
    if mask:
        out["mask"] = {"size": mask[0]}
        if mask[1] is not None:
            out["mask"]["keep_first"] = mask[1]
    return out


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=None, scaling=None):
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if vdim:
        out["vdim"] = vdim
    if base:
        out["rot"] = {"base": base, "dims": rot_dim}
        if scaling:
            out["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# SMALL: sizes that are no power of two; the loop in the middle of the stack, three passes; values wider and narrower
# than the keys; a window of an odd size beside an odd number of kept positions; a rotation over part of a head; a
# layer without feed-forward; a shared expert wider than the others and not a multiple of them; every expert chosen.
SMALL = {"architecture": "Mekuvik", "vocab": 211, "width": 72, "norm": {"eps": 3e-6}, "logit_scale": 0.7,
         "loop": {"start": 1, "stop": 4, "times": 3},
         "layers": [
             layer("attention", attention(6, 2, 14, 10, 0.31, (900.0, 6), (21, 3)), moe(24, 5, 2, 52)),
             layer("lightning", lightning(3, 10, 26, [0.5, 0.93, 0.998]), dense(44)),
             layer("latent_attention", latent(3, 12, 6, 16, 22, 18, 0.24, 700.0, (4.0, 64, 8.0, 1.5)), moe(20, 3, 3)),
             layer("attention", attention(4, 1, 18, 0, 0.2, (5000.0, 18), (9, 11)), None),
             layer("lightning", lightning(5, 6, 0, [0.0, 1.0, 0.7, 0.99, 0.9]), moe(16, 7, 1, 16))]}
# WIDE: heads of 64 and 128 values (the tensor-core kernels' sizes), also by padding, up to eight query heads per key
# head; windows across several key tiles and within one, kept positions across two pages and past a tile; states of 64
# and 128 key channels in the chunked form; the first layers looped, the last one too.
WIDE = {"architecture": "Mekuvik", "vocab": 300, "width": 128, "norm": {"eps": 1e-5}, "logit_scale": 1.6,
        "loop": {"start": 0, "stop": 4, "times": 2},
        "layers": [
            layer("attention", attention(8, 1, 64, 64, 0.11, (2000.0, 32), (150, 20)), moe(32, 6, 2, 64)),
            layer("lightning", lightning(2, 128, 72, [0.97, 0.9995]), dense(160)),
            layer("latent_attention", latent(4, 48, 16, 32, 64, 40, 0.12, 3000.0), moe(64, 4, 1, 40)),
            layer("attention", attention(2, 2, 128, 128, 0.08, (1e5, 128), (40, 140)), moe(48, 3, 1))]}
# BARE: the switches' other position: no loop, no scale of the logits, no window, no kept positions, no rotation, a key
# head per query head, one expert, heads and states of a few values, latents of one or two.
BARE = {"architecture": "Mekuvik", "vocab": 97, "width": 40, "norm": {"eps": 1e-5},
        "layers": [
            layer("latent_attention", latent(1, 4, 2, 0, 3, 1, 0.5), None),
            layer("attention", attention(2, 0, 8, 0, 0.4, None, (5, None)), moe(20, 1, 1)),
            layer("lightning", lightning(1, 1, 3, [0.8]), dense(24)),
            layer("attention", attention(3, 0, 6, 0, 0.45, (100.0, 2)), moe(12, 2, 2, 10))]}
MODELS = {"small": (SMALL, 61, 8, 1.0), "wide": (WIDE, 62, 16, 1.0), "bare": (BARE, 63, 4, 1.0),
          # score scales four times as large: which keys a query looks at decides its output
          "sharp": (SMALL, 64, 8, 4.0)}
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
            and (errors > 1.5).sum() <= max(1, 0.02 * len(errors)), (np.median(errors), np.quantile(errors, 0.95), (errors > 1.5).mean())


def sharpened(raw, factor):
    raw = json.loads(json.dumps(raw))
    for spec in raw["layers"]:
        if "scale" in spec["mixer"]:
            spec["mixer"]["scale"] *= factor
    return raw


def write_folder(folder, raw, seed, sharpen):
    """config.json + model.safetensors: bfloat16 matrices, float32 vectors (so
    that the engine and the plain side hold the same values). Projections are
    larger than the generator's (0.02) so that scores, gates and states move."""
    from metallix_b200.config import MekuvikConfig
    from metallix_b200.weights import random_tensors
    from metallix_b200.weights.safetensors_io import write_file
    config = MekuvikConfig.from_dict(sharpened(raw, sharpen))
    tensors = random_tensors(config, seed, dtype="bfloat16", norm_dtype="float32")
    for name, value in tensors.items():
        if value.dim() == 2:
            tensors[name] = (value.float() * (20.0 if name == "embed" else 4.0)).to(torch.bfloat16)
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
        folder = write_folder(str(tmp_path_factory.mktemp(f"mekuvik_{name}")), raw, seed, sharpen)
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
    from metallix_b200.config import ConfigError, MekuvikConfig, parse_config, resolve
    for raw in (SMALL, WIDE, BARE):
        config = parse_config(raw)
        assert isinstance(config, MekuvikConfig) and resolve(raw).kind == "mekuvik"
        assert MekuvikConfig.from_dict(config.to_dict()) == config
        assert json.loads(json.dumps(config.to_dict())) == config.to_dict()
        shapes, w = config.tensor_shapes(), raw["width"]
        assert shapes["embed"] == (raw["vocab"], w) and shapes["final.norm"] == (w,) and "head" not in shapes
        for index, spec in enumerate(raw["layers"]):
            base, mixer = f"l{index}", spec["mixer"]
            heads, dim = mixer["heads"], mixer["dim"]
            vdim = mixer.get("vdim") or dim
            assert shapes[f"{base}.norm1"] == (w,) and f"{base}.norm2" not in shapes
            if spec["type"] == "lightning":
                assert shapes[f"{base}.mix.k"] == (heads * dim, w) and shapes[f"{base}.mix.v"] == (heads * vdim, w)
                assert shapes[f"{base}.mix.norm"] == (heads * vdim,) and shapes[f"{base}.mix.g"] == (heads * vdim, w)
            elif spec["type"] == "attention":
                groups = mixer.get("kv_heads") or heads
                assert shapes[f"{base}.mix.k"] == (groups * dim, w) and shapes[f"{base}.mix.v"] == (groups * vdim, w)
                assert shapes[f"{base}.mix.q.norm"] == (heads * dim,) and shapes[f"{base}.mix.k.norm"] == (groups * dim,)
            else:
                assert shapes[f"{base}.mix.uq"] == (heads * (dim + mixer["rot_dim"]), mixer["q_rank"])
                assert shapes[f"{base}.mix.dkv"] == (mixer["kv_rank"] + mixer["rot_dim"], w)
                assert shapes[f"{base}.mix.uv"] == (heads * vdim, mixer["kv_rank"]) and shapes[f"{base}.mix.g"] == (heads * vdim, w)
            if spec["mlp"] is not None and spec["mlp"]["kind"] == "moe":
                assert shapes[f"{base}.mlp.router"] == (spec["mlp"]["router"]["experts"], w) and f"{base}.mlp.e0.gate" not in shapes
                assert (f"{base}.mlp.shared.up" in shapes) == ("shared" in spec["mlp"])
        model = config.to_model_spec()
        assert [(run.layer, run.join == 0) for run in model.order] == plain.layer_runs(raw)
        entries = [run.cache_entry() for run in model.order]
        assert len(set(entries)) == len(entries) and sorted(entries) == list(range(len(entries)))   # each pass its own
        assert (len(model.joins) == 1) == (raw.get("loop") is not None) and all(run.write_cache for run in model.order)
    once = json.loads(json.dumps(SMALL))
    once["loop"]["times"] = 1
    assert parse_config(once).to_model_spec().joins == () and len(parse_config(once).to_model_spec().order) == 5
    refusals = [
        ("UnsupportedLayerType", lambda c: c["layers"][1].update(type="delta")),
        ("InvalidGroupedQueryLayout", lambda c: c["layers"][0]["mixer"].update(kv_heads=4)),
        ("OddHeadDimension", lambda c: c["layers"][3]["mixer"].update(dim=17)),
        ("InvalidDecay", lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9])),
        ("InvalidDecay", lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, 1.5])),
        ("InvalidDecay", lambda c: c["layers"][1]["mixer"].update(decay=0.9)),
        ("Json", lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, None])),
        ("InvalidRotaryWidth", lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4)),
        ("InvalidRotaryWidth", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=16)),
        ("Json", lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1)),
        ("MissingDimension", lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)),
        ("MissingDimension", lambda c: c["layers"][2]["mixer"].update(q_rank=0)),
        ("UnsupportedFeedForward", lambda c: c["layers"][1]["mlp"].update(kind="relu")),
        ("Json", lambda c: c["layers"][0]["mlp"]["router"].update(top=6)),
        ("Json", lambda c: c["layers"][3]["mixer"].update(scale=-1.0)),
        ("Json", lambda c: c["loop"].update(stop=6)),
        ("Json", lambda c: c["loop"].update(start=4)),
        ("Json", lambda c: c.update(logit_scale="1")),
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


def test_random_weights_and_a_written_folder(tmp_path):
    from metallix_b200.config import MekuvikConfig
    from metallix_b200.weights import CheckpointError, load_tensors, random_tensors, write_model_folder
    config = MekuvikConfig.from_dict(SMALL)
    tensors = random_tensors(config, 3, dtype="float32")
    for name in ("l0.norm1", "l1.mix.norm", "l0.mix.q.norm", "l2.mix.dkv.norm", "final.norm"):
        assert abs(float(tensors[name].mean()) - 1.0) < 0.1, name
    assert abs(float(tensors["l1.mix.g"].mean())) < 0.01
    folder = write_model_folder(str(tmp_path / "m"), config, 3)
    assert set(load_tensors(folder, config)) == set(config.tensor_shapes())
    raw = json.loads(json.dumps(SMALL))
    raw["layers"][1]["mixer"]["vdim"] = 27
    with pytest.raises(CheckpointError):
        load_tensors(folder, MekuvikConfig.from_dict(raw))


def cpu_model(raw, dtype=torch.float32):
    from metallix_b200.config import MekuvikConfig
    from metallix_b200.engine.model import DecoderModel
    from metallix_b200.parts.registry import Runtime
    from metallix_b200.weights import random_tensors
    config = MekuvikConfig.from_dict(raw)
    tensors = random_tensors(config, 1, dtype="float32")
    return DecoderModel(config.to_model_spec(), dict(tensors), Runtime(device=torch.device("cpu"), dtype=dtype,
                                                                       max_positions=64)), tensors


def test_cache_needs_and_the_passes_entries():
    """Every pass of a looped layer has an entry of its own with the same needs; a window's need names its kept
    positions; a kept position without a window asks for nothing; a looped layer's weights count once per pass."""
    model, tensors = cpu_model(SMALL)
    needs = model.cache_needs()
    shape = lambda need: ("state", tuple(need.state_shape)) if need.kind == "state" else \
        (need.kind, need.kv_heads, need.head_dim, need.window, need.keep)
    want = {0: ("kv_pages", 2, 14, 21, 3), 1: ("state", (3, 26, 10)), 2: ("kv_pages", 3, 64, None, 0),
            3: ("kv_pages", 1, 18, 9, 11), 4: ("state", (5, 6, 6))}
    want.update({5: want[1], 6: want[2], 7: want[3], 8: want[1], 9: want[2], 10: want[3]})
    assert [shape(need) for need in needs] == [want[index] for index in range(11)]
    assert model.blocks[3].feed_forward is None and model.blocks[0].feed_forward_norm is None
    assert torch.allclose(model.final_norm.weight, tensors["final.norm"] * 0.7)
    once = json.loads(json.dumps(SMALL))
    once["loop"]["times"] = 1
    layers = sum(part.weight_bytes() for block in model.blocks[1:4] for part in (block.mixer, block.feed_forward)
                 if part is not None)
    assert model.weight_bytes() - cpu_model(once)[0].weight_bytes() == 2 * layers
    unmasked = json.loads(json.dumps(BARE))
    assert cpu_model(unmasked)[0].joins == [] and cpu_model(unmasked)[0].cache_needs()[1].window == 5
    # two windows of one size that keep different positions do not share pages
    twins = json.loads(json.dumps(BARE))
    twins["layers"][3]["mixer"].update(heads=2, dim=8, mask={"size": 5, "keep_first": 2})
    first, second = cpu_model(twins)[0].cache_needs()[1], cpu_model(twins)[0].cache_needs()[3]
    assert first.group_key() != second.group_key() and (first.keep, second.keep) == (0, 2)


def test_kept_positions_hold_their_pages():
    """Pages behind a window go back except those of the kept positions; the pages of kept positions go back with the
    request; under random orders nothing is lost or held twice."""
    from metallix_b200.csrc import build
    host = build.host()
    m = host.CacheManager([host.GroupConfig(4, 6, 12, 0, 5), host.GroupConfig(4, 0, 12)], 4)
    m.admit(1)
    m.reserve(1, 22)
    assert min(m.table(1, 0)) >= 0
    m.commit(1, 22)                 # the next query sees positions 17 .. 22 and 0 .. 4: pages 0, 1, 4, 5
    assert [page >= 0 for page in m.table(1, 0)] == [True, True, False, False, True, True]
    assert m.free_pages(0) == 8 and m.free_pages(1) == 6
    m.check_invariants()
    m.reserve(1, 8)
    m.rollback(1)
    assert m.free_pages(0) == 8
    m.fork(1, 2)
    m.check_invariants()
    m.release(1)
    assert [page >= 0 for page in m.table(2, 0)] == [True, True, False, False, True, True]
    m.release(2)
    assert m.free_pages(0) == 12
    rng = random.Random(4)
    for _ in range(30):
        page = rng.choice([1, 2, 4, 8])
        window, keep = rng.choice([1, 3, 7, 16]), rng.choice([0, 1, 4, 9, 40])
        m = host.CacheManager([host.GroupConfig(page, window, 64, 0, keep)], 3)
        held = {}
        for _ in range(60):
            name = rng.randrange(3)
            if name not in held:
                m.admit(name)
                held[name] = 0
            elif rng.random() < 0.1:
                m.release(name)
                del held[name]
            else:
                size = rng.randint(1, 9)
                if not m.fits([(name, size)]):
                    continue
                m.reserve(name, size)
                m.commit(name, size)
                held[name] += size
                table, count = m.table(name, 0), held[name]
                for p in range(count):
                    if p < keep or p > count - window:      # seen by the query at position `count`
                        assert table[p // page] >= 0, (page, window, keep, count, p)
                for index, entry in enumerate(table):
                    last = (index + 1) * page - 1
                    if index * page >= keep and last <= count - window and last < count:
                        assert entry < 0, (page, window, keep, count, index)
            m.check_invariants()
    with pytest.raises(ValueError):
        host.CacheManager([host.GroupConfig(4, 6, 12, 0, -1)], 4)


def test_heads_padded_to_a_size_the_tensor_cores_take():
    """The padded projections and norms give the same queries, keys, values and output as the given ones."""
    from metallix_b200.config import MekuvikConfig
    from metallix_b200.parts.attention import padded_heads
    from metallix_b200.parts.registry import Runtime, WeightStore
    rng = np.random.default_rng(2)
    config = MekuvikConfig.from_dict(SMALL)
    spec = config.layers[0].mixer.part("m", 72, 1e-3)
    shapes = config.layers[0].mixer.shapes("m", 72)
    tensors = {name: torch.tensor(rng.normal(size=shape)) for name, shape in shapes.items()}
    runtime = Runtime(device=torch.device("cpu"), dtype=torch.bfloat16, max_positions=8)
    wide, store = padded_heads(spec, WeightStore(dict(tensors)), runtime)
    assert wide["head_dim"] == wide["value_dim"] == 64 and wide["q_norm"]["size"] == 6 * 64
    x = rng.normal(size=(5, 72)) * 0.01
    get = lambda name: store.take(name).double().numpy()
    for which, heads in (("q", 6), ("k", 2)):
        given = plain.over_rms(x @ tensors[f"m.{which}"].numpy().T, 1e-3) * tensors[f"m.{which}.norm"].numpy()
        made = plain.over_rms(x @ get(f"m.{which}").T, wide[f"{which}_norm"]["eps"]) * get(f"m.{which}.norm")
        made = made.reshape(5, heads, 64)
        assert np.abs(made[:, :, :14] - given.reshape(5, heads, 14)).max() < 1e-6 and np.abs(made[:, :, 14:]).max() == 0.0
    value = (x @ get("m.v").T).reshape(5, 2, 64)
    assert np.abs(value[:, :, 10:]).max() == 0.0
    assert np.allclose(value[:, :, :10].reshape(5, 20), x @ tensors["m.v"].numpy().T, atol=1e-6)
    mixed = rng.normal(size=(5, 6, 64))
    assert np.allclose(mixed.reshape(5, -1) @ get("m.o").T, mixed[:, :, :10].reshape(5, -1) @ tensors["m.o"].numpy().T, atol=1e-5)
    for dtype, changed in ((torch.float32, {}), (torch.bfloat16, {"head_dim": 130, "value_dim": 130}),
                           (torch.bfloat16, {"head_dim": 64, "value_dim": 64})):      # left as they are
        given = type(spec)(spec.kind, dict(spec.params, **changed))
        same, _ = padded_heads(given, WeightStore({}), Runtime(device=torch.device("cpu"), dtype=dtype, max_positions=8))
        assert same is given


def random_model(raw, seed):
    from metallix_b200.config import MekuvikConfig
    rng = np.random.default_rng(seed)
    shapes = MekuvikConfig.from_dict(raw).tensor_shapes()
    return {name: 1.0 + rng.normal(size=shape) * 0.1 if len(shape) == 1 else rng.normal(size=shape) * 0.3
            for name, shape in shapes.items()}


def test_the_plain_side_in_pieces():
    """The plain implementation itself: logits do not change when more tokens
    follow; the recurrence in pieces, its states handed on, equals one run;
    single steps, the mask, the rotation and the experts by hand."""
    rng = np.random.default_rng(0)
    tensors = random_model(SMALL, 0)
    ids = random_ids(1, 40, 211)
    whole = plain.forward_logits(SMALL, tensors, ids)
    assert np.allclose(plain.forward_logits(SMALL, tensors, ids[:27]), whole[:27], atol=1e-9)
    h = rng.normal(size=(25, 72))
    run = lambda piece, states: plain.lightning(piece, tensors, "l1.mix", SMALL["layers"][1]["mixer"], 1e-6, states)
    once, _ = run(h, None)
    first, states = run(h[:2], None)
    second, states = run(h[2:11], states)
    third, _ = run(h[11:], states)
    assert np.allclose(np.concatenate([first, second, third]), once, atol=1e-12)
    k, v = np.array([[1.0, 2.0]]), np.array([[3.0, -1.0, 0.5]])
    out, state = plain.fading_memory(k, k, v, 0.5, np.ones((2, 3)))
    assert np.allclose(state, 0.5 + np.outer(k[0], v[0])) and np.allclose(out[0], state.T @ k[0])
    seen = plain.windowed_mask(12, {"size": 3, "keep_first": 2})
    assert [int(j) for j in np.nonzero(seen[9])[0]] == [0, 1, 7, 8, 9] and [int(j) for j in np.nonzero(seen[1])[0]] == [0, 1]
    assert [int(j) for j in np.nonzero(plain.windowed_mask(9, {"size": 2, "keep_first": 20})[6])[0]] == list(range(7))
    turned = plain.turn_pairs(np.array([[[1.0, 0.0, 5.0]]]), {"base": 10.0, "dims": 2}, [np.pi / 2])
    assert np.allclose(turned, [[[0.0, 1.0, 5.0]]])
    f, magnitude = plain.frequencies({"base": 700.0, "dims": 6, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.5}})
    assert np.isclose(magnitude, 0.1 * np.log(4.0) + 1.0) and np.isclose(f[0], 1.0) and np.isclose(f[2], 700.0 ** (-4 / 6) / 4.0)
    chosen, weights = plain.choose_experts(np.array([[1.0, 3.0, -2.0, 3.0]]), 3)
    assert chosen[0].tolist() == [1, 3, 0] and np.allclose(weights[0], plain.sigmoid(np.array([3.0, 3.0, 1.0])))
    one = {"m.e0.up": np.ones((1, 1)), "m.e0.down": np.ones((1, 1)), "m.router": np.zeros((1, 1))}
    got = plain.expert_mixture(np.array([[2.0]]), one, "m", {"router": {"experts": 1, "top": 1}})
    assert np.allclose(got, plain.gelu(np.array([[1.0]]))) and np.isclose(plain.gelu(np.array([1.0]))[0], 0.8413447460685429)


def test_the_models_of_these_tests_show_a_window_kept_positions_a_state_and_a_pass(folders):
    """What the tests below can see: on the plain side, a window one position
    longer or shorter, one kept position more or fewer, a state lost at one
    position, one pass fewer, passes that do not meet the embedding output,
    weights behind the experts or renormalized, and values that are not gated
    each move the logits by far more than the bound the engine is held to."""
    _, config, tensors, _ = folders["sharp"]
    tensors = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    ids = random_ids(40, 75, config["vocab"])
    base = plain.forward_logits(config, tensors, ids)
    gap = lambda logits, first=0: np.abs(logits - base)[first:].max()

    def changed(change):
        other = json.loads(json.dumps(config))
        change(other)
        return plain.forward_logits(other, tensors, ids)

    masks = lambda c, key, by: [spec["mixer"]["mask"].update({key: spec["mixer"]["mask"][key] + by})
                                for spec in c["layers"] if spec["type"] == "attention"]
    lost = np.concatenate([plain.forward_logits(config, tensors, ids[:60]), plain.forward_logits(config, tensors, ids[60:])])
    ungated = dict(tensors, **{"l2.mix.g": tensors["l2.mix.g"] * 0.0})
    gaps = {"longer": gap(changed(lambda c: masks(c, "size", 1))), "shorter": gap(changed(lambda c: masks(c, "size", -1))),
            "more kept": gap(changed(lambda c: masks(c, "keep_first", 1))),
            "fewer kept": gap(changed(lambda c: masks(c, "keep_first", -1))), "state": gap(lost, 60),
            "passes": gap(changed(lambda c: c["loop"].update(times=2))),
            "scaling": gap(changed(lambda c: c["layers"][2]["mixer"]["rot"].pop("scaling"))),
            "decay": gap(changed(lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.93, 0.99]))),
            "gate": gap(plain.forward_logits(config, ungated, ids))}
    runs, mixture, choose = plain.layer_runs, plain.expert_mixture, plain.choose_experts
    try:
        plain.layer_runs = lambda c: [(index, False) for index, _ in runs(c)]
        gaps["meeting"] = gap(plain.forward_logits(config, tensors, ids))
        plain.layer_runs = runs
        plain.choose_experts = lambda z, top: (lambda c, w: (c, w / w.sum(axis=-1, keepdims=True)))(*choose(z, top))
        gaps["renormalized"] = gap(plain.forward_logits(config, tensors, ids))
        plain.choose_experts = lambda z, top: (choose(z, top)[0], np.ones((z.shape[0], top)))
        gaps["unweighed"] = gap(plain.forward_logits(config, tensors, ids))
    finally:
        plain.layer_runs, plain.expert_mixture, plain.choose_experts = runs, mixture, choose
    assert min(gaps.values()) > 20 * TOL_SHARP, gaps


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
@pytest.mark.parametrize("dtype, form", [(torch.float32, "tokens"), (torch.bfloat16, "tokens"), (torch.float32, "steps"),
                                         (torch.bfloat16, "steps"), (torch.bfloat16, "chunks")])
@pytest.mark.parametrize("heads, dim, vdim", [(3, 16, 40), (2, 128, 64), (1, 8, 8), (2, 64, 104), (1, 96, 32), (4, 40, 136),
                                              (2, 12, 20), (1, 1, 3), (1, 200, 33)])
def test_lightning_attention(dtype, form, heads, dim, vdim):
    """Linear attention with a constant decay over request rows of unequal
    length in one launch (a single token, a padding row, rows of exactly one and
    two chunks and one more), continued twice from the state the launch before
    left, against the plain recurrence in one piece. Among the decays are 0 and
    1; the first token's value is large and the last token's query is the first
    token's key, so that what the first token wrote is what the last one reads."""
    from metallix_b200 import ops
    if (form == "chunks" and (dim % 8 or vdim % 8 or dim > 128)) or (form == "steps" and (dim % 4 or dim > 128)):
        with pytest.raises(ops.KernelError):
            wide = torch.zeros((2, heads * (2 * dim + vdim)), dtype=dtype, device="cuda")
            one = dev([0], torch.int32)
            ops.lightning_attention(wide, (0, heads * dim, 2 * heads * dim), torch.ones(heads, device="cuda"),
                                    torch.zeros((1, heads, vdim, dim), device="cuda"), one, one, one, heads, dim, vdim, form=form)
        return
    rng = np.random.default_rng(heads * dim + vdim)
    pieces = [[64, 1, 0, 5, 130], [1, 1, 0, 65, 2], [9, 3, 0, 1, 128]]
    slots = [2, 0, 1, 3, 5]
    totals = [sum(p[row] for p in pieces) for row in range(5)]
    decay = rounded(np.array([0.999, 0.0, 1.0, 0.6])[:heads], torch.float32)
    seq = []
    for total in totals:
        first = np.where(np.arange(total) == 0, 32.0, 1.0)[:, None]
        q_rows, k_rows = rng.normal(size=(total, heads * dim)), rng.normal(size=(total, heads * dim))
        if total > 30:
            q_rows[-1] = k_rows[0]
        seq.append({"q": rounded(q_rows, dtype), "k": rounded(k_rows, dtype),
                    "v": rounded(rng.normal(size=(total, heads * vdim)) * first, dtype)})
    state = torch.full((7, heads, vdim, dim), 3.0, device="cuda")      # S transposed: a column's channels side by side
    for slot in slots:
        state[slot].zero_()
    got, done = [[] for _ in totals], [0] * 5
    for lengths in pieces:
        starts = rows_of(lengths)
        pack = lambda key: np.concatenate([seq[row][key][done[row]:done[row] + n] for row, n in enumerate(lengths)])
        columns = 8 + heads * (2 * dim + vdim)
        wide = dev(np.concatenate([np.ones((sum(lengths), 8)), pack("q"), pack("k"), pack("v"),
                                   np.ones((sum(lengths), 8 + -columns % 8))], axis=1), dtype)
        out = ops.lightning_attention(wide, (8, 8 + heads * dim, 8 + 2 * heads * dim), dev(decay), state, dev(starts, torch.int32),
                                      dev(lengths, torch.int32), dev(slots, torch.int32), heads, dim, vdim,
                                      longest=max(lengths), form=form)
        ops.check_status("cuda")
        assert float((wide[:, :8] - 1.0).abs().max()) == 0.0 and float((wide[:, columns:] - 1.0).abs().max()) == 0.0
        for row, n in enumerate(lengths):
            got[row].append(out[starts[row]:starts[row] + n].double().cpu().numpy())
            done[row] += n
    assert float(state[4].min()) == 3.0 and float(state[6].min()) == 3.0       # untouched slots
    assert float(state[1].abs().max()) == 0.0                                  # a padding row's slot
    act = lambda x: rounded(plain.silu(x), dtype)
    tolerance = 2e-4 if dtype == torch.float32 else 3e-3 if form == "chunks" else 2e-3
    for row, total in enumerate(totals):
        if not total:
            continue
        q, k = (act(seq[row][key]).reshape(total, heads, dim) for key in "qk")
        v = act(seq[row]["v"]).reshape(total, heads, vdim)
        for head in range(heads):
            want, last = plain.fading_memory(q[:, head], k[:, head], v[:, head], decay[head])
            have = np.concatenate(got[row])[:, head * vdim:(head + 1) * vdim]
            assert np.abs(have - want).max() < tolerance * max(1.0, np.abs(want).max()), (row, head)
            kept = state[slots[row], head].double().cpu().numpy().T
            assert np.abs(kept - last).max() < tolerance * max(1.0, np.abs(last).max()), (row, head)
            if total > 30 and decay[head] > 0.9 and dim > 1:      # without the first token's write the last output is another
                again, _ = plain.fading_memory(q[1:, head], k[1:, head], v[1:, head], decay[head])
                close = tolerance * max(1.0, np.abs(want[-1]).max())
                assert np.abs(have[-1] - want[-1]).max() < close and np.abs(again[-1] - want[-1]).max() > 3 * close


@gpu
@pytest.mark.parametrize("dtype, head_dim, heads, kv_heads, context, page, window, keep", [
    (torch.bfloat16, 64, 8, 2, 700, 16, 150, 5), (torch.bfloat16, 128, 4, 4, 1500, 16, 129, 128),
    (torch.bfloat16, 128, 2, 1, 600, 32, 40, 33), (torch.bfloat16, 64, 6, 6, 2600, 16, 2200, 1), (torch.bfloat16, 64, 4, 2, 400, 4, 61, 30),
    (torch.bfloat16, 64, 4, 1, 300, 16, 7, 200), (torch.bfloat16, 256, 4, 1, 500, 16, 100, 20), (torch.float32, 64, 4, 2, 500, 8, 65, 9),
    (torch.float32, 128, 8, 1, 300, 16, 128, 140), (torch.float32, 24, 3, 1, 200, 4, 31, 3), (torch.bfloat16, 40, 6, 3, 300, 8, 64, 17),
    (torch.bfloat16, 64, 4, 2, 500, 16, 100, 0)])
def test_a_window_beside_kept_positions_in_every_attention_kernel(dtype, head_dim, heads, kv_heads, context, page, window, keep):
    """Queries that see a window and the first few positions, in the general
    kernel, the split-key decode kernels and both tensor-core prompt kernels,
    with edges inside and at the border of key tiles. The block table has holes
    between the kept pages and the window, and what the cache holds outside the
    seen pages is not a number. Four queries look for one key each: the window's
    last and the one before it, the last kept position and the one behind it."""
    from metallix_b200 import ops
    rng = np.random.default_rng(head_dim + context + keep)
    scale, tail = 0.15, 40
    group, first = heads // kv_heads, context - tail
    keys = rng.normal(size=(context, kv_heads, head_dim)) * 0.5
    values = rng.normal(size=(context, kv_heads, head_dim))
    q = rng.normal(size=(tail, heads, head_dim)) * 0.3
    spots = {5: first + 5 - window + 1, 8: first + 8 - window, 20: keep - 1, 21: keep}
    spots = {t: key for t, key in spots.items() if key >= 0}
    for t, key in spots.items():
        keys[key] = rng.normal(size=(kv_heads, head_dim)) * (0.5 * 64 ** 0.25 / head_dim ** 0.25)
        q[t] = np.repeat(keys[key], group, axis=0) * (12.0 / (scale * (keys[key] ** 2).sum(axis=-1).mean()))
    keys, values, q = rounded(keys, dtype), rounded(values, dtype), rounded(q, dtype)
    pages = -(-context // page)
    order = rng.permutation(pages + 2)[:pages]
    pool = torch.full((pages + 2, 2, kv_heads, page, head_dim), float("nan"), dtype=dtype, device="cuda")
    lowest = first - window + 1       # nothing between the kept positions and this one is seen by any query here
    holes = np.array(order)
    for p in range(pages):
        span = slice(p * page, min((p + 1) * page, context))
        if span.start >= keep and span.stop <= lowest:
            holes[p] = -1             # given back: another request's, and whatever that left
            continue
        n = span.stop - span.start
        pool[order[p], 0, :, :n] = dev(keys[span].transpose(1, 0, 2), dtype)
        pool[order[p], 1, :, :n] = dev(values[span].transpose(1, 0, 2), dtype)
    positions = np.arange(first, context)
    k_all, v_all = np.repeat(keys, group, axis=1), np.repeat(values, group, axis=1)

    def attended(size, kept):
        out = np.zeros((tail, heads, head_dim))
        for t, p in enumerate(positions):
            j = np.arange(p + 1)
            visible = (p - j < size) | (j < kept)
            s = np.einsum("hd,jhd->hj", q[t], k_all[:p + 1]) * scale
            out[t] = np.einsum("hj,jhd->hd", plain.softmax(s, np.broadcast_to(visible, s.shape)), v_all[:p + 1])
        return out

    want = attended(window, keep)
    tolerance = 3e-5 if dtype == torch.float32 else 3e-2
    inner = [t for t, key in spots.items() if key < first]
    for other, t in ((attended(window - 1, keep), 5), (attended(window + 1, keep), 8), (attended(window, keep - 1), 20),
                     (attended(window, keep + 1), 21)):
        if t in inner and not (t == 21 and keep > lowest) and not (t == 20 and keep - 1 >= lowest) and not (t in (5, 8) and spots[t] < keep):
            assert np.abs(other[t] - want[t]).max() > 10 * tolerance, t       # an edge one position off would show
    tables = dev(holes[None, :], torch.int32)
    out = torch.empty((tail, heads, head_dim), dtype=dtype, device="cuda")
    ops.paged_attention_tile(dev(q, dtype), pool, out, tables, dev([0, 0, 0], torch.int32), dev([0, 16, 32], torch.int32),
                             dev([16, 16, tail - 32], torch.int32), dev(positions, torch.int32), scale, window, keep=keep)
    ops.check_status("cuda")
    assert np.abs(out.double().cpu().numpy() - want).max() < tolerance
    if ops.decode_attention_supported(head_dim, heads, kv_heads, dtype):
        w = rounded(rng.normal(size=(96, heads * head_dim)) * 0.05, torch.bfloat16)
        try:
            for resident in (444, 0, 2):       # a block per tile or few blocks that walk over tiles
                ops.set_decode_resident_blocks(resident, max(resident, 2))
                for t in (0, 5, 8, 20, 21, tail - 1):      # each as a single decoded token behind its context
                    one = torch.empty((1, heads, head_dim), dtype=dtype, device="cuda")
                    lists = (tables, dev([0], torch.int32), dev([0], torch.int32), dev(positions[t:t + 1], torch.int32))
                    ops.paged_attention_decode(dev(q[t:t + 1], dtype), pool, one, *lists, scale, int(positions[t]) + 1,
                                               window=window, keep=keep)
                    ops.check_status("cuda")
                    assert np.abs(one.double().cpu().numpy()[0] - want[t]).max() < tolerance, (t, resident)
                    if dtype == torch.bfloat16 and head_dim <= 128:
                        parts = ops.paged_attention_decode_project(dev(q[t:t + 1], dtype), pool, *lists, scale,
                                                                   int(positions[t]) + 1, dev(w, dtype), window=window, keep=keep)
                        ops.check_status("cuda")
                        assert np.abs(parts.sum(0).double().cpu().numpy()[0] - want[t].reshape(-1) @ w.T).max() < 6e-2, (t, resident)
        finally:
            ops.set_decode_resident_blocks(444)
    if ops.flash_prefill_supported(head_dim, heads, kv_heads, dtype):
        try:
            for kernel in ("tcgen05", "mma"):
                if kernel == "tcgen05" and not ops.flash_prefill_tcgen05_supported(head_dim, heads, kv_heads, page, dtype):
                    continue
                for shares in (None, 3):
                    ops.KEY_SHARES = shares
                    out.zero_()
                    ops.flash_prefill(dev(q, dtype), pool, out, tables, dev([0], torch.int32), dev([0], torch.int32),
                                      dev([tail], torch.int32), dev(positions, torch.int32), scale, window, kernel=kernel,
                                      longest_context=context, keep=keep)
                    ops.check_status("cuda")
                    assert np.abs(out.double().cpu().numpy() - want).max() < tolerance, (kernel, shares)
        finally:
            ops.KEY_SHARES = None


@gpu
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("parts, part_size", [(1, 60), (3, 20), (4, 7), (1, 9000), (2, 512)])
def test_a_gate_behind_a_norm_in_parts(out_dtype, parts, part_size):
    from metallix_b200 import ops
    rng = np.random.default_rng(part_size)
    tokens, width, eps = 6, parts * part_size, 1e-4
    x = rounded(rng.normal(size=(tokens, width)) * 0.1, torch.float32)
    w = rounded(1.0 + rng.normal(size=width) * 0.3, torch.float32)
    tolerance = 3e-5 if out_dtype == torch.float32 else 8e-3      # of the largest value
    for gate_type in (torch.float32, torch.bfloat16):
        gate = rounded(rng.normal(size=(tokens, width)) * 2.0, gate_type)
        for before in (3, 8):      # rows that vectors divide, and not
            wide = dev(np.concatenate([np.zeros((tokens, before)), gate, np.zeros((tokens, 8))], axis=1), gate_type)
            for name, act in (("silu", plain.silu), ("sigmoid", plain.sigmoid)):
                got = ops.gated_norm(dev(x), dev(w), wide[:, before:before + width], parts, eps, out_dtype, activation=name,
                                     behind=True)
                want = plain.over_rms(x.reshape(tokens, parts, part_size), eps).reshape(tokens, width) * w * act(gate)
                assert np.abs(got.double().cpu().numpy() - want).max() < tolerance * np.abs(want).max(), name


@gpu
@pytest.mark.parametrize("size", [72, 128, 4096])
def test_a_pass_meets_the_embedding_output(size):
    """x += m (a + b) + c with its norm, and the join through each kind of
    thing that may be pending, ahead of the next norm or alone; the embedding
    output is left as it is."""
    from metallix_b200 import ops
    from metallix_b200.config.spec import PartSpec
    from metallix_b200.parts.block import PairSum
    from metallix_b200.parts.norm import RMSNorm
    from metallix_b200.parts.registry import Runtime, WeightStore, build_part, settle
    rng = np.random.default_rng(size)
    rows, eps = 5, 1e-5
    runtime = Runtime(device=torch.device("cuda"), dtype=torch.bfloat16, max_positions=16)
    join = build_part("join", PartSpec("add_first", {"hidden_size": size}), WeightStore({}), runtime)
    x, c = (rounded(rng.normal(size=(rows, size)), torch.float32) for _ in range(2))
    w = rounded(1.0 + rng.normal(size=size) * 0.2, torch.float32)
    norm = RMSNorm(torch.tensor(w), eps, runtime)
    for kind in ("none", "tensor", "pair", "one of a pair", "joined"):
        a, b = rounded(rng.normal(size=(rows, size)), torch.bfloat16), rounded(rng.normal(size=(rows, size)), torch.float32)
        pending, added = None, 0.0
        if kind == "tensor":
            pending, added = dev(a, torch.bfloat16), a
        elif kind == "pair":
            pending, added = PairSum(dev(a, torch.bfloat16), dev(b), 0.5), 0.5 * (a + b)
        elif kind == "one of a pair":
            pending, added = PairSum(dev(a, torch.bfloat16), None, 1.0), a
        elif kind == "joined":
            pending, added = PairSum(None, dev(b), 1.0, extra=dev(a)), a + b
        want = x + added + c
        for alone in (True, False):
            stream, first = dev(x), dev(c)
            residual, left = join.forward(stream, pending, first, 1)
            if alone:
                settle(residual, left)
            else:
                normed = norm.add_forward(residual, left, torch.float32)
                assert np.abs(normed.double().cpu().numpy() - plain.over_rms(want, eps) * w).max() < 2e-5
            assert np.abs(residual.double().cpu().numpy() - want).max() < 1e-5, kind
            assert np.array_equal(first.double().cpu().numpy(), c)
    stream = dev(x)       # the stream is still the embedding output itself
    residual, left = join.forward(stream, None, stream, 1)
    settle(residual, left)
    assert np.abs(residual.double().cpu().numpy() - 2 * x).max() < 1e-5 and np.array_equal(stream.double().cpu().numpy(), x)
    stream = dev(x)
    y = ops.pair_add_rmsnorm(stream, dev(x), None, 2.0, dev(w), None, eps, torch.float32, c=dev(c))
    assert np.abs(y.double().cpu().numpy() - plain.over_rms(3 * x + c, eps) * w).max() < 2e-5


@gpu
def test_the_exact_gelu_in_every_kernel_that_holds_it():
    """The pass of its own, the tensor-core product's epilogue with and
    without a weight per row, against the error function itself, out to where
    the tanh form differs."""
    from metallix_b200 import ops, tensor_core
    rng = np.random.default_rng(7)
    grid = np.linspace(-8.0, 8.0, 4001)
    got = ops.gelu(dev(grid)).double().cpu().numpy()
    assert np.abs(got - plain.gelu(rounded(grid, torch.float32))).max() < 1e-6
    tanh_form = 0.5 * grid * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (grid + 0.044715 * grid ** 3)))
    assert np.abs(tanh_form - plain.gelu(grid)).max() > 1e-4
    for count in (4000, 4001):      # whole vectors, and not
        half = rounded(grid[:count], torch.bfloat16)
        assert np.abs(ops.gelu(dev(half, torch.bfloat16)).double().cpu().numpy() - plain.gelu(half)).max() < 2e-2
    a, w = rounded(rng.normal(size=(200, 64)), torch.bfloat16), rounded(rng.normal(size=(96, 64)) * 0.2, torch.bfloat16)
    got = tensor_core.gemm_gelu(dev(a, torch.bfloat16), dev(w, torch.bfloat16)).double().cpu().numpy()
    assert np.abs(got - plain.gelu(a @ w.T)).max() < 3e-2
    rows = 384
    a = rounded(rng.normal(size=(rows, 64)), torch.bfloat16)
    scale = rounded(rng.uniform(0.05, 1.0, size=rows), torch.float32)
    stacked = rounded(rng.normal(size=(3 * 40, 64)) * 0.3, torch.bfloat16)
    for given in (None, scale):
        got = tensor_core.gemm_grouped(dev(a, torch.bfloat16), dev(stacked, torch.bfloat16), dev([2, 0, 1], torch.int32), 3,
                                       tensor_core.GELU, row_scale=None if given is None else dev(given))
        for tile, group in enumerate((2, 0, 1)):
            at = slice(tile * 128, (tile + 1) * 128)
            product = a[at] @ stacked[group * 40:(group + 1) * 40].T * (1.0 if given is None else given[at, None])
            assert np.abs(got[at].double().cpu().numpy() - plain.gelu(product)).max() < 3e-2
    with pytest.raises(ops.KernelError):
        tensor_core.gemm_grouped(dev(a, torch.bfloat16), dev(stacked, torch.bfloat16), dev([2, 0, 1], torch.int32), 3,
                                 tensor_core.RELU_SQUARED, row_scale=dev(scale))


@gpu
@pytest.mark.parametrize("experts, top", [(6, 2), (8, 1), (3, 3), (1, 1), (64, 6), (300, 5)])
def test_router_whose_scores_are_the_weights(experts, top):
    from metallix_b200 import ops
    rng = np.random.default_rng(experts * top)
    tokens = 37
    logits = rounded(rng.normal(size=(tokens, experts)) * 3.0, torch.float32)
    chosen, weights, dense_weights, on_identity = ops.route_experts(dev(logits), torch.zeros(experts, device="cuda"), experts, top,
                                                                    scores="sigmoid", normalized=False, always=2)
    want_chosen, want_weights = plain.choose_experts(logits, top)
    assert np.array_equal(chosen.cpu().numpy()[:, :top], want_chosen)
    assert np.array_equal(chosen.cpu().numpy()[:, top:], np.tile([experts, experts + 1], (tokens, 1)))
    assert np.abs(weights.double().cpu().numpy()[:, :top] - want_weights).max() < 1e-6
    assert float((weights[:, top:] - 1.0).abs().max()) == 0.0 and float(on_identity.abs().max()) == 0.0
    assert np.abs(dense_weights.sum(dim=1).double().cpu().numpy() - want_weights.sum(axis=1)).max() < 1e-5


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens, shared", [(1, 24), (1, 0), (5, 40), (300, 80), (5, 0), (300, 95), (5, 8), (1700, 120)])
def test_experts_weighed_at_their_input(dtype, tokens, shared):
    """Experts of the exact gelu through the part itself, row by row and
    grouped, with a shared expert narrower than the others, as wide, a multiple
    and none. A weight outside of the gelu is another number: the plain side
    shows it."""
    from metallix_b200.config.mekuvik import WeighedExperts
    from metallix_b200.parts.registry import Runtime, WeightStore, build_part
    rng = np.random.default_rng(tokens + shared)
    hidden, ff, experts, top = 64, 40, 5, 2
    typed = WeighedExperts(ff=ff, experts=experts, top=top, shared_ff=shared)
    tensors = {k: rounded(rng.normal(size=shape) * (0.3 if k.endswith("down") else 0.12), torch.bfloat16)
               for k, shape in typed.shapes("m", hidden).items()}
    part = build_part("feed_forward", typed.part("m", hidden), WeightStore({k: torch.tensor(v) for k, v in tensors.items()}),
                      Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=16))
    assert part.always == {0: 0, 8: 0, 24: 0, 40: 1, 80: 2, 95: 3, 120: 3}[shared] and (part.shared is None) == (shared not in (8, 24))
    h = rounded(rng.normal(size=(tokens, hidden)), dtype)
    got = part.forward(dev(h, dtype), None).double().cpu().numpy()
    want = plain.expert_mixture(h, tensors, "m", typed.to_dict())
    chosen, weights = plain.choose_experts(h @ tensors["m.router"].T, top)
    behind = want.copy()
    for t in range(min(tokens, 5)):
        for e, w in zip(chosen[t], weights[t]):
            up, down = tensors[f"m.e{e}.up"], tensors[f"m.e{e}.down"]
            behind[t] += w * plain.gelu_ff(h[t:t + 1], up, down)[0] - plain.gelu_ff(w * h[t:t + 1], up, down)[0]
    scale = max(1.0, np.abs(want).max())
    assert np.abs(behind - want).max() > 0.03 * scale
    errors = np.abs(got - want).max(axis=1)
    if dtype == torch.float32:
        assert errors.max() < 1e-4 * scale
    else:       # a close call of the router may go the other way for a token in a hundred
        assert np.quantile(errors, 0.97) < 1.2e-2 * scale


def part_context(tokens, page, dtype):
    from metallix_b200.parts.registry import StepContext
    ints = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")
    return ints, StepContext(device=torch.device("cuda"), dtype=dtype, num_tokens=tokens, num_requests=1,
                             positions=ints(list(range(tokens))), token_request=ints([0] * tokens), request_slots=ints([0]),
                             request_offsets=[0, tokens], request_positions=[0])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mode", ["heads", "latent"])
@pytest.mark.parametrize("sizes", [(3, 12, 6, 16, 22, 18), (4, 48, 16, 32, 64, 40), (2, 40, 24, 64, 17, 33), (2, 96, 32, 128, 48, 64)])
def test_gated_latent_attention_in_both_cache_modes(dtype, mode, sizes):
    """The mixer alone: queries and the latent through their norms, the gate
    inside the attention kernels (rows per head, padded) or behind the widening,
    stretched wavelengths."""
    from metallix_b200 import ops
    from metallix_b200.config.mekuvik import GatedLatentAttention
    from metallix_b200.config.spec import PartSpec
    from metallix_b200.parts.registry import CacheView, Runtime, WeightStore, build_part
    rng = np.random.default_rng(sizes[1])
    heads, dim, rot, vdim, q_rank, kv_rank = sizes
    raw = latent(heads, dim, rot, vdim, q_rank, kv_rank, 0.6 / (dim + rot) ** 0.5, 500.0, (4.0, 32, 6.0, 1.0))
    typed = GatedLatentAttention.from_dict(raw, "mixer")
    hidden, tokens, page, eps = 80, 37, 8, 1e-5
    tensors = {name: rounded(1.0 + rng.normal(size=shape) * 0.1 if len(shape) == 1 else rng.normal(size=shape) * 0.25, torch.bfloat16)
               for name, shape in typed.shapes("m", hidden).items()}
    spec = typed.part("m", hidden, eps)
    spec = PartSpec(spec.kind, dict(spec.params, cache_mode=mode))
    part = build_part("mixer", spec, WeightStore({k: torch.tensor(v, dtype=torch.float32) for k, v in tensors.items()}),
                      Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=64))
    x = rounded(rng.normal(size=(tokens, hidden)), dtype)
    need = part.cache_need()
    ints, ctx = part_context(tokens, page, dtype)
    pages = -(-tokens // page)
    view = CacheView(need, pool=torch.zeros((pages, need.planes, need.kv_heads, page, need.head_dim), dtype=dtype, device="cuda"),
                     block_tables=ints([list(range(pages))]), slots=ints(list(range(tokens))))
    got = part.forward(dev(x, dtype), ctx, view).double().cpu().numpy()
    ops.check_status("cuda")
    want = plain.latent_attention(x, tensors, "m", raw, eps)
    ungated = plain.latent_attention(x, dict(tensors, **{"m.g": tensors["m.g"] * 0.0}), "m", raw, eps)
    tolerance = (1e-4 if dtype == torch.float32 else 5e-2) * max(1.0, np.abs(want).max())
    assert np.abs(got - want).max() < tolerance and np.abs(ungated - want).max() > 5 * tolerance


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot", [(6, 2, 14, 10, 6), (4, 1, 40, 96, 40), (2, 2, 96, 80, 32), (8, 1, 64, 64, 16),
                                                             (3, 3, 136, 136, 2), (2, 1, 130, 64, 130)])
def test_attention_with_norms_over_the_projections_and_padded_heads(dtype, heads, kv_heads, dim, vdim, rot):
    """The mixer alone, prompts of 50 tokens under a window beside kept
    positions, with heads that are padded in bfloat16 and heads that are not."""
    from metallix_b200 import ops
    from metallix_b200.config.mekuvik import KeptWindowAttention
    from metallix_b200.parts.registry import CacheView, Runtime, WeightStore, build_part
    rng = np.random.default_rng(dim)
    raw = attention(heads, kv_heads, dim, vdim, 0.5 / dim ** 0.5, (300.0, rot), (13, 4))
    typed = KeptWindowAttention.from_dict(raw, "mixer")
    hidden, tokens, page, eps = 64, 50, 8, 1e-2
    tensors = {name: rounded(1.0 + rng.normal(size=shape) * 0.1 if len(shape) == 1 else rng.normal(size=shape) * 0.1, torch.bfloat16)
               for name, shape in typed.shapes("m", hidden).items()}
    part = build_part("mixer", typed.part("m", hidden, eps),
                      WeightStore({k: torch.tensor(v, dtype=torch.float32) for k, v in tensors.items()}),
                      Runtime(device=torch.device("cuda"), dtype=dtype, max_positions=64))
    padded = dtype == torch.bfloat16 and max(dim, vdim) <= 128
    assert part.head_dim == ((64 if max(dim, vdim) <= 64 else 128) if padded else dim) and part.flash == padded
    x = rounded(rng.normal(size=(tokens, hidden)), dtype)
    need = part.cache_need()
    ints, ctx = part_context(tokens, page, dtype)
    pages = -(-tokens // page)
    view = CacheView(need, pool=torch.zeros((pages, 2, need.kv_heads, page, need.head_dim), dtype=dtype, device="cuda"),
                     block_tables=ints([list(range(pages))]), slots=ints(list(range(tokens))))
    got = part.forward(dev(x, dtype), ctx, view).double().cpu().numpy()
    ops.check_status("cuda")
    want = plain.window_attention(x, tensors, "m", raw, eps)
    assert np.abs(got - want).max() < (1e-4 if dtype == torch.float32 else 3e-2) * max(1.0, np.abs(want).max())


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
    (over more tokens than the small windows hold), and in portions of changing
    size down to two tokens (and one)."""
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
@pytest.mark.parametrize("dim", [64, 24])
def test_a_key_at_either_side_of_a_windows_edge_and_of_the_last_kept_position(folders, dtype, dim):
    """Attention through the engine's cache where one earlier token decides
    what a late one answers, if it is seen: the projections of the one layer are
    made so that the last token's query is that token's key and nobody else's.
    The token stands at a kept position (the first, the last, at a page's
    border), just behind them, just inside and just outside of the window, in a
    prompt and decoded alone behind portions; with another token in its place
    the logits are far away where it is seen, and the same where it is not."""
    from metallix_b200.config import MekuvikConfig
    from metallix_b200.engine import Engine, StepEntry
    rng = np.random.default_rng(12)
    window, keep, last = 70, 21, 200
    raw = {"architecture": "Mekuvik", "vocab": 64, "width": dim, "norm": {"eps": 1e-6}, "logit_scale": 2.0,
           "layers": [layer("attention", attention(2, 1, dim, 0, 14.0 / dim, (50.0, 2), (window, keep)), None)]}
    tensors = random_model(raw, 4)
    tensors["embed"] = rng.normal(size=(64, dim))
    tensors["embed"][:, :2] = 0.0        # the rotated pair: where a key stands does not matter
    tensors["embed"][62] = np.concatenate([np.zeros(2), np.roll(tensors["embed"][63, 2:], 1)])
    turn = np.eye(dim)
    turn[2:, 2:] = np.roll(np.eye(dim - 2), 1, axis=0)      # q of 63 = k of 62
    tensors["l0.mix.q"] = np.concatenate([turn] * 2)
    tensors["l0.mix.k"] = np.eye(dim)
    tensors["l0.mix.v"] = np.eye(dim) * 3.0
    tensors["l0.mix.o"] = np.concatenate([np.roll(np.eye(dim), 5, axis=0), np.zeros((dim, dim))], axis=1)
    for name in ("l0.norm1", "final.norm", "l0.mix.q.norm", "l0.mix.k.norm"):
        tensors[name] = np.ones_like(tensors[name])
    tensors = {name: rounded(value, torch.bfloat16) for name, value in tensors.items()}
    seen_at = {0: True, 15: True, 16: True, keep - 1: True, keep: False, 64: False, last - window: False,
               last - window + 1: True, last - 8: True, last - 1: True}
    engine = Engine(MekuvikConfig.from_dict(raw), {k: torch.tensor(v, dtype=torch.float32) for k, v in tensors.items()},
                    dtype=dtype, page_tokens=16, num_pages=16, max_requests=1)
    for early, seen in seen_at.items():
        ids = [int(t) for t in rng.integers(1, 60, size=last)]
        ids[early] = 62
        ids.append(63)
        want = plain.forward_logits(raw, tensors, ids)[-1]
        other = plain.forward_logits(raw, tensors, ids[:early] + [7] + ids[early + 1:])[-1]
        tolerance = 2e-4 if dtype == "float32" else 3e-1
        assert (np.abs(want - other).max() > 8 * tolerance) == seen and (seen or np.abs(want - other).max() < 1e-9), early
        for sizes in ([last + 1], [last, 1], [100, 64, 36, 1], [3] * 66 + [2, 1]):
            logits, at = None, 0
            for size in sizes:
                logits = engine.step([StepEntry("a", ids[at:at + size], [size - 1])])
                at += size
            engine.check()
            assert np.abs(logits[0].double().cpu().numpy() - want).max() < tolerance, (early, sizes)
            table = engine.manager.table(engine._ids["a"], 0)
            assert [page >= 0 for page in table[:2]] == [True, True] and table[4] < 0      # kept pages stay, others went back
            engine.release("a")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_captured_steps(folders, dtype):
    """Three requests decoded together for 160 steps (captured graphs), one of
    them leaving on the way and another joining with a prompt: the states of
    every pass, the pages behind the windows and the kept ones stay each
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
    ids = random_ids(3, 60, config["vocab"])
    other = ids[:42] + random_ids(4, 18, config["vocab"])
    engine = make_engine(folders, name, "float32", pages=64)
    engine.step([StepEntry("p", ids[:42], [])])
    engine.fork("p", "c")
    a = engine.step([StepEntry("p", ids[42:], list(range(18))), StepEntry("c", other[42:], list(range(18)))])
    engine.check()
    want = np.concatenate([plain.forward_logits(config, tensors, ids)[42:], plain.forward_logits(config, tensors, other)[42:]])
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
