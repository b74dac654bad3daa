"""Kipizen without a GPU: configuration, module construction, the registry, and properties of the plain implementation the GPU
tests lean on."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import kipizen_ref as ref
import kipizen_util as util
from onyxia_b200 import checkpoint, ir, kipizen, models

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _folder(tmp_path, config, w):
    with open(tmp_path / "config.json", "w") as f:
        json.dump(config, f)
    checkpoint.write_safetensors(str(tmp_path / "model.safetensors"), checkpoint.Weights.from_bf16(
        {k: checkpoint.Weights.from_f32({k: v}).bf16_bits(k) for k, v in w.items()}))
    return str(tmp_path)


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
def test_a_model_folder_becomes_a_module(tmp_path, name):
    config, w = util.model(name)
    folder = _folder(tmp_path, config, w)
    assert {k: v.shape for k, v in w.items()} == kipizen.tensor_shapes(kipizen.KipizenConfig.from_dict(config))
    mixers = [l["mixer"] for l in config["layers"]]
    own = [i for i, m in enumerate(mixers) if "decay" not in m and m.get("kv_from") is None]
    for dtype in ("bfloat16", "float32"):
        m = models.load_module(folder, dtype)
        m.validate()
        ins = m.input_names()
        assert {"input_ids", "seq_info", "logit_rows"} <= set(ins) and ("page_table" in ins) == bool(own)
        state = [n for n in ins if n.startswith(("pages.", "slots."))]
        assert sorted(m.output_names()) == sorted(["logits"] + ["updated." + n for n in state])
        assert [n for n in state if n.startswith("pages.")] == [f"pages.{i}.{part}" for i in own for part in ("keys", "values")]
        ops = m.node_ops()
        assert ops.count("onyxia.PagedKVAttention") == len(own)
        assert ops.count("onyxia.SharedKVAttention") == sum(m.get("kv_from") is not None for m in mixers)
        assert ops.count("onyxia.LightningAttention") == sum("decay" in m for m in mixers)
        assert ops.count("onyxia.MixtureOfExperts") == sum(l["mlp"] is not None for l in config["layers"])
    if own:
        a = mixers[own[0]]
        assert m.eval_input_shape(ins.index(f"pages.{own[0]}.values"), {"num_pages": 5}) == (5, a["kv_heads"], 64, a["vdim"])


def test_configuration_is_read():
    c = kipizen.KipizenConfig.from_dict(util.CONFIGS["mixed"])
    assert (c.vocab, c.width, c.eps, c.embed_scale) == (131, 64, 1e-5, 3.0)
    a = c.layers[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.softcap, a.scale, a.kv_from) == (4, 2, 16, 24, 90, 20.0, 0.5, 0)
    assert (a.rot_dims, a.rot_base, a.rot_factor) == (8, 500.0, 2.0) and c.layers[3].experts is None
    assert c.layers[1].mixer.decay == [0.7, 0.999, 0.95] and c.layers[2].experts == kipizen.ExpertsConfig(5, 3, 24)


def _changed(path, value):
    c = copy.deepcopy(util.CONFIGS["mixed"])
    at = c["layers"]
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return c


@pytest.mark.parametrize("path,value,message", [
    ([0, "type"], "serial", "serial"), ([0, "mlp", "kind"], "dense", "dense"), ([0, "mixer", "heads"], 5, "5 query heads"),
    ([0, "mixer", "rot", "dims"], 7, "pairs"), ([0, "mixer", "rot", "dims"], 18, "pairs"), ([2, "mixer", "kv_from"], 1, "no keys of its own"),
    ([2, "mixer", "kv_from"], 4, "no keys of its own"), ([2, "mixer", "dim"], 32, "differ in size"), ([1, "mixer", "decay"], [0.5], "1 decays for 3"),
    ([0, "mlp", "router", "top"], 9, "9 of 8"), ([0, "mixer", "mask", "size"], 0, "window")])
def test_bad_configurations_are_refused(path, value, message):
    with pytest.raises(ValueError, match=message):
        kipizen.KipizenConfig.from_dict(_changed(path, value))


def test_bad_weights_are_refused():
    config, w = util.model("mixed")
    cfg = kipizen.KipizenConfig.from_dict(config)
    for name in ("l0.mix.k.b", "l1.mix.norm", "l4.mlp.e3.up", "l0.mlp.router.b", "head"):
        short = dict(w)
        del short[name]
        with pytest.raises(KeyError, match=name):
            kipizen.build(cfg, checkpoint.Weights.from_f32(short))
        with pytest.raises(ValueError):
            kipizen.build(cfg, checkpoint.Weights.from_f32(dict(w, **{name: w[name][:-1]})))
    with pytest.raises(ValueError, match="bf16 or f32"):
        kipizen.build(cfg, checkpoint.Weights.from_f32(w), ir.F16)


def test_turns_and_powers():
    t = kipizen.turns_per_position(10, 300.0, 4.0).astype(np.float64).sum(axis=0)
    assert np.allclose(t * 2 * math.pi, [300.0 ** (-i / 5) / 4.0 for i in range(5)], rtol=1e-13, atol=0)
    d = kipizen.decay_table([0.999, 0.0, 1.0])
    assert d.shape == (3, kipizen.CHUNK + 2) and d[0, 64] == np.float32(0.999 ** 64) and d[0, 65] == np.float32(0.999 - 1.0)
    assert d[1, :2].tolist() == [1.0, 0.0] and d[1, 65] == -1.0 and (d[2, :65] == 1.0).all()


def test_random_weights_build():
    c = kipizen.KipizenConfig.from_dict(util.CONFIGS["wide"])
    w = kipizen.random_weights(c)
    assert {n: w.shape(n) for n in w.names()} == kipizen.tensor_shapes(c)
    kipizen.build(c, w).validate()


# ── the plain implementation ──
def test_plain_window_edges():
    r = np.random.default_rng(3)
    T, window = 30, 7
    q, k, v = r.standard_normal((T, 4, 8)), r.standard_normal((T, 2, 8)), r.standard_normal((T, 2, 5))
    base = ref.attention(q, k, v, 0.3, 5.0, window)
    for j in (0, 1, 12, 29):
        v2 = v.copy()
        v2[j] += 1.0
        moved = np.abs(ref.attention(q, k, v2, 0.3, 5.0, window) - base).max(axis=(1, 2))
        sees = (np.arange(T) >= j) & (np.arange(T) < j + window)
        assert (moved[~sees] == 0).all() and (moved[sees] > 1e-4).all()


def test_plain_sink_and_softcap():
    q, k, v = np.ones((1, 1, 4)), np.ones((1, 1, 4)), np.ones((1, 1, 2))
    s = 3.0 * math.tanh(2.0 / 3.0)
    assert np.allclose(ref.attention(q, k, v, 0.5, 3.0, 4), math.exp(s) / (1 + math.exp(s)))
    assert np.allclose(ref.attention(q, k, v, 0.5, 3.0, 4, sink=False), 1.0)


def test_plain_rotation_keeps_lengths_and_distances():
    r = np.random.default_rng(1)
    q, k = np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0), np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0)
    a, b = ref.rotate(q, 50.0, 6, 2.0), ref.rotate(k, 50.0, 6, 2.0)
    assert np.allclose((a ** 2).sum(axis=2), (q ** 2).sum(axis=2)) and np.array_equal(a[..., 6:], q[..., 6:])
    assert np.allclose([(a[i, 0] * b[i - 3, 0]).sum() for i in range(3, 20)], (a[3, 0] * b[0, 0]).sum())
    assert not np.allclose(a[5], q[5])


def test_plain_state_and_experts():
    r = np.random.default_rng(2)
    q, k, v = r.standard_normal((9, 2, 4)), r.standard_normal((9, 2, 4)), r.standard_normal((9, 2, 3))
    decay = np.array([0.5, 0.9])
    o = ref.decayed_state(q, k, v, decay)
    for h in range(2):
        want = sum(decay[h] ** (8 - j) * (q[8, h] @ k[j, h]) * v[j, h] for j in range(9))
        assert np.allclose(o[8, h], want)
    chosen, weight = ref.route(np.array([[1.0, 0.0], [0.0, 1.0]]), np.array([[0.0, 1.0], [2.0, 0.0], [1.0, 3.0]]), np.array([0.0, 0.0, 0.5]), 2)
    assert chosen.tolist() == [[1, 2], [2, 0]] and np.allclose(weight.sum(axis=1), 1)
    assert np.allclose(weight[0], [math.exp(0.5) / (1 + math.exp(0.5)), 1 / (1 + math.exp(0.5))])


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
def test_small_models_choose_experts_clearly(name):
    """The routers of the test models read levels that are far apart next to the rounding of bf16."""
    config, w = util.model(name)
    coded = max([l["mlp"]["router"]["experts"] for l in config["layers"] if l["mlp"]], default=0)
    _, streams = ref.forward(config, w, util.tokens(name, 40), every_layer=True)
    x = w["embed"][util.tokens(name, 40)] * config["embedding"]["scale"]
    for s in streams:
        assert np.allclose(s[:, :coded], x[:, :coded], rtol=1e-12)
    gaps = np.diff(np.sort(x[:, :coded], axis=1), axis=1)
    assert gaps.min() > 2.0 / coded


def test_command_line_lists_it():
    r = subprocess.run([sys.executable, "-m", "onyxia_b200", "models"], cwd=ROOT, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=120)
    assert r.returncode == 0 and "Kipizen" in r.stdout
