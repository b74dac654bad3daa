"""Zusitar without a GPU: configuration, module construction, the registry, and properties of the plain implementation the GPU
tests lean on."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import zusitar_ref as ref
import zusitar_util as util
from onyxia_b200 import checkpoint, ir, models, zusitar

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
    assert {k: v.shape for k, v in w.items()} == zusitar.tensor_shapes(zusitar.ZusitarConfig.from_dict(config))
    kinds = [config["layers"][i]["type"] for i, _ in ref.layer_runs(config)]
    names = {"mamba1": ["slots.{}.conv", "slots.{}.state"], "latent_attention": ["pages.{}.latents"], "attention": ["pages.{}.keys", "pages.{}.values"]}
    for dtype in ("bfloat16", "float32"):
        m = models.load_module(folder, dtype)
        m.validate()
        ins = m.input_names()
        state = [n for n in ins if n.startswith(("pages.", "slots."))]
        assert state == [s.format(n) for n, k in enumerate(kinds) for s in names[k]]
        assert {"input_ids", "seq_info", "logit_rows"} <= set(ins) and ("page_table" in ins) == any(k != "mamba1" for k in kinds)
        assert sorted(m.output_names()) == sorted(["logits"] + ["updated." + n for n in state])
        ops = m.node_ops()
        assert [ops.count("onyxia." + o) for o in ("SelectiveScan", "LatentAttention", "PagedKVAttention")] == [kinds.count(k) for k in names]
        assert ops.count("onyxia.MixtureOfExperts") == sum((config["layers"][i]["mlp"] or {}).get("kind") == "moe" for i, _ in ref.layer_runs(config))
    n = kinds.index("latent_attention") if "latent_attention" in kinds else None
    if n is not None:
        m_ = config["layers"][ref.layer_runs(config)[n][0]]["mixer"]
        assert m.eval_input_shape(ins.index(f"pages.{n}.latents"), {"num_pages": 5}) == (5, 1, 64, m_["kv_rank"] + m_["rot_dim"])


def test_configuration_is_read():
    c = zusitar.ZusitarConfig.from_dict(util.CONFIGS["mixed"])
    assert (c.vocab, c.width, c.eps, c.embed_scale, c.loop) == (131, 96, 1e-5, 3.0, (1, 4, 2))
    assert c.runs() == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None), (5, None)]
    assert c.layers[0].mixer == zusitar.MambaConfig(96, 8, 4, 4) and c.layers[1].mlp == zusitar.DenseConfig(72) and c.layers[3].mlp is None
    assert c.layers[1].mixer == zusitar.LatentConfig(4, 16, 8, 24, 24, 32, 0.5, 700.0)
    assert c.layers[2].mixer == zusitar.AttentionConfig(4, 2, 16, 24, 0.7, 8, 500.0, 6.0) and c.layers[4].mixer.softcap == 0.0
    assert c.layers[0].mlp == zusitar.ExpertsConfig(8, 2, 40, 1.5, 1.3, 4, 2, 56, 0.8) and c.layers[4].mlp.groups == 0
    c = zusitar.ZusitarConfig.from_dict(util.CONFIGS["odd"])
    assert c.runs() == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None), (2, None), (3, None)]
    assert c.layers[2].mixer.rot_dims == 0 and c.layers[2].mlp.shared_ff == 0
    assert zusitar.ZusitarConfig.from_dict(util.CONFIGS["wide"]).runs() == [(i, None) for i in range(5)]


def _changed(path, value):
    c = copy.deepcopy(util.CONFIGS["mixed"])
    at = c
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return c


@pytest.mark.parametrize("path,value,message", [
    (["layers", 0, "type"], "serial", "serial"), (["layers", 0, "mlp", "kind"], "sparse", "sparse"), (["layers", 2, "mixer", "heads"], 5, "5 query heads"),
    (["layers", 2, "mixer", "rot", "dims"], 7, "pairs"), (["layers", 2, "mixer", "rot", "dims"], 18, "pairs"), (["layers", 1, "mixer", "rot", "dims"], 4, "4 of the 8"),
    (["layers", 0, "mlp", "router", "top"], 5, "5 of 8"), (["layers", 0, "mlp", "router", "groups", "count"], 3, "3 groups"),
    (["layers", 0, "mlp", "router", "groups", "keep"], 5, "5 of 4"), (["loop", "stop"], 9, "loop"), (["loop", "start"], 4, "loop"), (["loop", "times"], 0, "0 times")])
def test_bad_configurations_are_refused(path, value, message):
    with pytest.raises(ValueError, match=message):
        zusitar.ZusitarConfig.from_dict(_changed(path, value))


def test_bad_weights_are_refused():
    config, w = util.model("mixed")
    cfg = zusitar.ZusitarConfig.from_dict(config)
    for name in ("embed", "loop.step", "l0.mix.A_log", "l0.mix.conv", "l0.mlp.shared.up", "l0.mlp.e3.down", "l1.mix.uk", "l1.mix.dkv.norm", "l1.norm2b", "l2.mix.sink",
                 "l2.mix.o.b", "l2.mlp.router", "l3.norm1b", "final.norm"):
        short = dict(w)
        del short[name]
        with pytest.raises(KeyError, match=name):
            zusitar.build(cfg, checkpoint.Weights.from_f32(short))
        with pytest.raises(ValueError):
            zusitar.build(cfg, checkpoint.Weights.from_f32(dict(w, **{name: w[name][:-1]})))
    with pytest.raises(ValueError, match="bf16 or f32"):
        zusitar.build(cfg, checkpoint.Weights.from_f32(w), ir.F16)


def test_random_weights_build():
    c = zusitar.ZusitarConfig.from_dict(util.CONFIGS["mixed"])
    w = zusitar.random_weights(c)
    assert {n: w.shape(n) for n in w.names()} == zusitar.tensor_shapes(c)
    zusitar.build(c, w).validate()


# ── the plain implementation ──
def test_plain_sink_and_softcap():
    q, k, v = np.ones((1, 2, 4)), np.ones((1, 1, 4)), np.ones((1, 1, 2))
    s, sinks = 3.0 * math.tanh(2.0 / 3.0), np.array([0.5, -1.0])
    got = ref.attention(q, k, v, 0.5, 3.0, sinks)[0]
    assert np.allclose(got, (math.exp(s) / (np.exp(sinks) + math.exp(s)))[:, None])
    assert np.allclose(ref.attention(q, k, v, 0.5, 3.0), 1.0)


@pytest.mark.parametrize("interleaved", [False, True])
def test_plain_rotation_keeps_lengths_and_distances(interleaved):
    r = np.random.default_rng(1)
    q, k = np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0), np.repeat(r.standard_normal((1, 1, 10)), 20, axis=0)
    a, b = ref.rotate(q, 50.0, 6, interleaved), ref.rotate(k, 50.0, 6, interleaved)
    assert np.allclose((a ** 2).sum(axis=2), (q ** 2).sum(axis=2)) and np.array_equal(a[..., 6:], q[..., 6:])
    assert np.allclose([(a[i, 0] * b[i - 3, 0]).sum() for i in range(3, 20)], (a[3, 0] * b[0, 0]).sum())
    u, v = (0, 1) if interleaved else (0, 3)  # the fastest pair turns by one radian per position
    assert np.allclose(a[2, 0, u], q[0, 0, u] * math.cos(2) - q[0, 0, v] * math.sin(2))


def test_plain_scan_and_convolution():
    r = np.random.default_rng(2)
    x, dt, B, C = r.standard_normal((9, 3)), r.uniform(0.1, 1, (9, 3)), r.standard_normal((9, 4)), r.standard_normal((9, 4))
    A, D = -r.uniform(0.1, 2, (3, 4)), r.standard_normal(3)
    y = ref.selective_scan(x, dt, A, B, C, D)
    for c in range(3):
        want = D[c] * x[8, c] + sum((np.exp(A[c] * dt[j + 1:, c].sum()) * dt[j, c] * x[j, c] * B[j]) @ C[8] for j in range(9))
        assert np.allclose(y[8, c], want)
    w, b = r.standard_normal((3, 4)), r.standard_normal(3)
    u = ref.causal_conv(x, w, b)
    assert np.allclose(u[0], b + w[:, 3] * x[0]) and np.allclose(u[5], b + sum(w[:, k] * x[2 + k] for k in range(4)))


def test_plain_experts_of_the_best_groups():
    z = np.array([[2.0, -3.0, 1.9, 1.8, 1.0, 1.2, 3.0, -9.0]])  # groups by their two best: (2, 3) > (4, 5) > (0, 1) ~ (6, 7)
    c = {"experts": 8, "top": 3, "scale": 2.0, "groups": {"count": 4, "keep": 2}}
    chosen, weight = ref.route(z, np.eye(8), c)
    s = ref.sigmoid(z[0, [2, 3, 5]])
    assert chosen.tolist() == [[2, 3, 5]] and np.allclose(weight, 2 * s / s.sum())
    assert ref.route(z, np.eye(8), dict(c, groups=None))[0].tolist() == [[6, 0, 2]]
    assert ref.route(z, np.eye(8), dict(c, groups={"count": 4, "keep": 4}))[0].tolist() == [[6, 0, 2]]


@pytest.mark.parametrize("name", sorted(util.CONFIGS))
def test_small_models_choose_experts_clearly(name):
    """The routers of the test models read levels that are far apart next to the rounding of bf16, whatever passes of the loop and
    norms have made of their scale."""
    config, w = util.model(name)
    routers, coded = util._routers(config)
    toks = util.tokens(name, 40)
    _, streams = ref.forward(config, w, toks, every_layer=True)
    x = w["embed"][toks] * config["embedding"]["scale"]
    start, stop, times = [config["loop"][k] for k in ("start", "stop", "times")] if config["loop"] else (0, 0, 1)
    for (i, t), s in zip(ref.layer_runs(config), streams):
        passes = 1 + t if t is not None else times if i >= stop else 1
        assert np.allclose(s[:, :coded], passes * x[:, :coded], rtol=1e-12)
    for (experts, groups), at in routers.items():
        own = np.sort(x[:, at: at + experts].reshape(len(x), groups, -1), axis=2)
        assert np.diff(np.sort(x[:, at: at + experts], axis=1), axis=1).min() > 2.0 / experts
        if groups > 1 and experts > groups:
            first, second = np.sort(own[:, :, -1], axis=1), np.sort(own[:, :, -2], axis=1)
            assert (second[:, 1:] - first[:, :-1]).min() > 2.0 / experts


def test_command_line_lists_it():
    r = subprocess.run([sys.executable, "-m", "onyxia_b200", "models"], cwd=ROOT, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=120)
    assert r.returncode == 0 and "Zusitar" in r.stdout
