"""Mufevik without a GPU: configuration, module construction, the registry, and properties of the plain implementation the GPU
tests lean on."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import mufevik_ref as ref
import mufevik_util as util
from onyxia_b200 import checkpoint, ir, models, mufevik

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
    ranks = {f"l{i}.mix.right.{n}" for i in range(len(config["layers"])) for n in ("a1", "a2")}  # their size is the checkpoint's own
    shapes = mufevik.tensor_shapes(mufevik.MufevikConfig.from_dict(config))
    assert {k: v.shape for k, v in w.items() if k not in ranks} == {k: v for k, v in shapes.items() if k not in ranks} and set(w) == set(shapes)
    kinds = [l["type"] for l in config["layers"]]
    names = {"delta": ["slots.{}.conv", "slots.{}.state"], "parallel": ["pages.{}.keys", "pages.{}.values", "slots.{}.state"]}
    for dtype in ("bfloat16", "float32"):
        m = models.load_module(folder, dtype)
        m.validate()
        ins = m.input_names()
        state = [n for n in ins if n.startswith(("pages.", "slots."))]
        assert state == [s.format(n) for n, k in enumerate(kinds) for s in names[k]]
        assert {"input_ids", "seq_info", "logit_rows"} <= set(ins) and ("page_table" in ins) == ("parallel" in kinds)
        assert sorted(m.output_names()) == sorted(["logits"] + ["updated." + n for n in state])
        ops = m.node_ops()
        assert ops.count("onyxia.GatedDeltaRule") == kinds.count("delta") and ops.count("onyxia.PagedKVAttention") == ops.count("onyxia.GatedLinearAttention") == kinds.count("parallel")
        assert ops.count("onyxia.MixtureOfExperts") == sum(l["mlp"] is not None for l in config["layers"])
    for i, l in enumerate(config["layers"]):
        c = l["mixer"] if l["type"] == "delta" else l["mixer"]["right"]
        assert m.eval_input_shape(ins.index(f"slots.{i}.state"), {"num_slots": 5}) == (5, c["heads"], c["dim"], c["vdim"])


def test_configuration_is_read():
    c = mufevik.MufevikConfig.from_dict(util.CONFIGS["mixed"])
    assert (c.vocab, c.width, c.eps, c.streams, c.logit_scale) == (131, 96, 1e-3, 2, 0.7)
    assert c.layers[0].mixer == mufevik.ParallelConfig(mufevik.AttentionConfig(4, 2, 16, 24, 0.5, 8, 500.0), mufevik.LinearConfig(3, 16, 8, 4.0))
    assert c.layers[1].mixer == mufevik.DeltaConfig(4, 2, 16, 24, 4) and c.layers[2].mixer.taps == 2 and c.layers[2].experts is None
    assert c.layers[0].experts == mufevik.ExpertsConfig(8, 3, 40, 4, 2, 56) and c.layers[1].experts.shared_ff == 0
    assert c.layers[4].mixer.left.rot_dims == 0 and c.layers[4].mixer.right.tau == 16.0
    c = mufevik.MufevikConfig.from_dict(util.CONFIGS["odd"])
    assert c.streams == 1 and c.layers[1].experts == mufevik.ExpertsConfig(6, 3, 7)


def _changed(path, value):
    c = copy.deepcopy(util.CONFIGS["mixed"])
    at = c
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return c


@pytest.mark.parametrize("path,value,message", [
    (["layers", 0, "type"], "serial", "serial"), (["layers", 0, "mlp", "kind"], "dense", "dense"), (["layers", 0, "mixer", "left", "heads"], 5, "5 heads"),
    (["layers", 1, "mixer", "heads"], 3, "3 heads over 2"), (["layers", 0, "mixer", "left", "rot", "dims"], 7, "pairs"), (["layers", 0, "mixer", "left", "rot", "dims"], 18, "pairs"),
    (["layers", 0, "mixer", "right", "tau"], 0, "1 / 0"), (["layers", 0, "mlp", "router", "top"], 5, "5 of 8"), (["layers", 0, "mlp", "router", "groups", "count"], 3, "3 groups"),
    (["layers", 0, "mlp", "router", "groups", "keep"], 5, "5 of 4"), (["streams"], 0, "0 streams")])
def test_bad_configurations_are_refused(path, value, message):
    with pytest.raises(ValueError, match=message):
        mufevik.MufevikConfig.from_dict(_changed(path, value))


def test_bad_weights_are_refused():
    config, w = util.model("mixed")
    cfg = mufevik.MufevikConfig.from_dict(config)
    for name in ("embed", "head", "l0.norm1", "l0.hc1.mix", "l0.hc2.in", "l0.hc2.out", "l0.mix.left.talk", "l0.mix.left.temp", "l0.mix.left.out", "l0.mix.right.a1", "l0.mix.right.a2.b",
                 "l0.mix.right.norm", "l0.mlp.correction", "l0.mlp.shared.sg", "l0.mlp.e3.down", "l1.mix.A_log", "l1.mix.q.conv", "l1.mix.dt_bias", "l1.mix.norm", "l1.mix.b", "final.norm"):
        short = dict(w)
        del short[name]
        with pytest.raises(KeyError, match=name):
            mufevik.build(cfg, checkpoint.Weights.from_f32(short))
        with pytest.raises(ValueError):
            mufevik.build(cfg, checkpoint.Weights.from_f32(dict(w, **{name: w[name][:-1] if w[name].shape else np.ones(2)})))
    with pytest.raises(ValueError, match="bf16 or f32"):
        mufevik.build(cfg, checkpoint.Weights.from_f32(w), ir.F16)


def test_random_weights_build():
    c = mufevik.MufevikConfig.from_dict(util.CONFIGS["mixed"])
    w = mufevik.random_weights(c)
    assert {n: w.shape(n) for n in w.names()} == mufevik.tensor_shapes(c)
    mufevik.build(c, w).validate()


# ── the plain implementation ──
def test_plain_talking_heads():
    r = np.random.default_rng(0)
    q, k, v = r.standard_normal((6, 4, 8)), r.standard_normal((6, 2, 8)), r.standard_normal((6, 2, 3))
    temp = r.uniform(0.5, 2, 4)
    alone = ref.talking_attention(q, k, v, 0.5, temp)
    assert np.allclose(ref.talking_attention(q, k, v, 0.5, temp, np.eye(4)), alone)
    s = np.exp(0.5 * temp[3] * k[:, 1] @ q[5, 3])
    assert np.allclose(alone[5, 3], s @ v[:, 1] / s.sum())
    # head 0 with head 3's weights still has its own values
    talk = np.eye(4)
    talk[0] = [0, 0, 0, 2.0]
    assert np.allclose(ref.talking_attention(q, k, v, 0.5, temp, talk)[5, 0], 2 * s @ v[:, 0] / s.sum())


def test_plain_rotation_keeps_lengths_and_distances():
    r = np.random.default_rng(1)
    q, k = np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0), np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0)
    a, b = ref.rotate(q, 50.0, 6), ref.rotate(k, 50.0, 6)
    assert np.allclose((a ** 2).sum(axis=2), (q ** 2).sum(axis=2)) and np.array_equal(a[..., 6:], q[..., 6:])
    assert np.allclose([(a[i, 0] * b[i - 3, 0]).sum() for i in range(3, 20)], (a[3, 0] * b[0, 0]).sum())
    assert np.allclose(a[2, 0, 0], q[0, 0, 0] * math.cos(2) - q[0, 0, 3] * math.sin(2))


def test_plain_linear_attention_and_delta_rule():
    r = np.random.default_rng(2)
    q, k, v = r.standard_normal((9, 2, 4)), r.standard_normal((9, 2, 4)), r.standard_normal((9, 2, 3))
    alpha = r.uniform(0.2, 1, (9, 2, 4))
    o = ref.gated_linear_attention(q, k, v, alpha)
    want = sum((q[8, 1] * k[j, 1] * alpha[j + 1:, 1].prod(axis=0)).sum() * v[j, 1] for j in range(9))
    assert np.allclose(o[8, 1], want)
    k = ref.unit(k)
    o = ref.gated_delta_rule(k, k, v, np.ones((9, 2)), np.ones((9, 2)))
    assert np.allclose(o, v, atol=1e-5)  # a unit key with a whole step reads what it wrote
    still = ref.gated_delta_rule(q, k, v, np.ones((9, 2)), np.zeros((9, 2)))
    assert np.allclose(still, 0.0)
    w = r.standard_normal((3, 4))
    x = r.standard_normal((9, 3))
    u = ref.causal_conv(x, w)
    assert np.allclose(u[0], w[:, 3] * x[0]) and np.allclose(u[5], sum(w[:, i] * x[2 + i] for i in range(4)))


def test_plain_choice_of_experts():
    z = np.log(np.array([[0.3, 0.1, 0.2, 0.15, 0.05, 0.2]]))
    c = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, weight = ref.route(z, np.eye(6), np.array([-1.0, -9.0, -0.8, -2.0, -3.0, -3.0]), c)
    assert chosen.tolist() == [[2, 3]] and np.allclose(weight, [[0.2, 0.15]])  # the second group has the best corrected expert
    assert ref.route(z, np.eye(6), np.zeros(6), dict(c, groups=None))[0].tolist() == [[0, 2]]


def test_plain_streams():
    r = np.random.default_rng(3)
    x, w = r.standard_normal((3, 5, 4)), {"in": r.standard_normal(3), "out": r.standard_normal(3), "mix": r.standard_normal((3, 3))}
    got = ref.hyper(x, w, lambda u: 2 * u)
    u = w["in"][0] * x[0] + w["in"][1] * x[1] + w["in"][2] * x[2]
    assert np.allclose(got[1], w["mix"][0, 1] * x[0] + w["mix"][1, 1] * x[1] + w["mix"][2, 1] * x[2] + w["out"][1] * 2 * u)


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
def test_small_models_choose_experts_clearly(name, monkeypatch):
    """The routers of the test models read levels that are far apart next to the rounding of bf16."""
    config, w = util.model(name)
    gaps, route = [], ref.route

    def spy(h, router, correction, c):
        z = h @ router.T
        gaps.append(np.diff(np.sort(z, axis=1), axis=1).min() / np.abs(z).max())
        return route(h, router, correction, c)

    monkeypatch.setattr(ref, "route", spy)
    ref.forward(config, w, util.tokens(name, 60))
    assert min(gaps) > 2.0 ** -7


def test_command_line_lists_it():
    r = subprocess.run([sys.executable, "-m", "onyxia_b200", "models"], cwd=ROOT, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=120)
    assert r.returncode == 0 and "Mufevik" in r.stdout
