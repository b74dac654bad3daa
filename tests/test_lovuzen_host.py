"""Lovuzen without a GPU: configuration, checkpoint files, module construction, the registry, and properties of the plain
implementation the GPU tests lean on."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import lovuzen_ref as ref
import lovuzen_util as util
from onyxia_b200 import checkpoint, ir, lovuzen, models

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("rows,far", [(2, 5), (7, 30), (16, 64), (32, 128), (24, 500), (9, 10)])
def test_distance_rows_match_the_bucket_rule(rows, far):
    got = lovuzen.distance_rows(rows, far)
    assert got.tolist() == [ref.distance_bucket(n, rows, far) for n in range(far + 1)]
    assert got[far] == rows - 1 and all(ref.distance_bucket(n, rows, far) == rows - 1 for n in (far, far + 1, 10 * far))
    assert (np.diff(got) >= 0).all()


def test_distance_rows_on_exact_row_edges():
    # 16 rows to 128: row 8 + k starts at 8 · 2^(k/2), a whole number for even k
    got = lovuzen.distance_rows(16, 128)
    for k in (0, 2, 4, 6):
        n = 8 * 2 ** (k // 2)
        assert got[n] == 8 + k and got[n - 1] == (7 + k)
    # 32 rows to 16 · 3^4: quarters of the upper half start at powers of three
    got = lovuzen.distance_rows(32, 16 * 81)
    for k in range(4):
        n = 16 * 3 ** k
        assert got[n] == 16 + 4 * k and got[n - 1] == 15 + 4 * k


def test_distance_bias_layout():
    table = np.arange(12, dtype=np.float32).reshape(6, 2)
    b = lovuzen.distance_bias(table, 20)
    assert b.shape == (2, 21)
    for n in range(21):
        assert b[1, n] == table[ref.distance_bucket(n, 6, 20), 1]


def test_safetensors_round_trip(tmp_path):
    r = np.random.default_rng(0)
    w = checkpoint.Weights({"a": ("BF16", r.integers(0, 2 ** 16, (3, 5)).astype(np.uint16) & 0xBF7F),
                            "b.c": ("F32", r.standard_normal(7).astype(np.float32)), "t": ("I32", np.arange(4, dtype=np.int32)),
                            "none": ("F32", np.zeros((0, 3), np.float32))})
    path = str(tmp_path / "model.safetensors")
    checkpoint.write_safetensors(path, w)
    got = checkpoint.read_safetensors(path)
    assert got.names() == w.names()
    for n in w.names():
        assert got._get(n)[0] == w._get(n)[0] and np.array_equal(got._get(n)[1], w._get(n)[1])
    assert np.array_equal(got.f32("a").view(np.uint32), w._get("a")[1].astype(np.uint32) << 16)
    assert np.array_equal(got.bf16_bits("a"), w._get("a")[1])
    with pytest.raises(KeyError, match="missing"):
        got.f32("missing")
    with open(path, "r+b") as f:
        f.truncate(os.path.getsize(path) - 1)
    with pytest.raises(ValueError, match="does not fit"):
        checkpoint.read_safetensors(path)


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
    assert {k: v.shape for k, v in w.items()} == lovuzen.tensor_shapes(lovuzen.LovuzenConfig.from_dict(config), util.BIAS_ROWS[name])
    for dtype in ("bfloat16", "float32"):
        m = models.load_module(folder, dtype)
        m.validate()
        ins = m.input_names()
        assert ins[:4] == ["input_ids", "seq_info", "page_table", "logit_rows"] and m.output_names()[0] == "logits"
        assert sorted(m.output_names()[1:]) == sorted("updated." + n for n in ins[4:])
        assert m.node_ops().count("onyxia.PagedAttention") == len(config["layers"])
        i = ins.index("slots.0.conv")
        r = config["layers"][0]["mixer"]["right"]
        assert m.eval_input_shape(i, {"num_slots": 5}) == (5, r["conv"], r["width"])


def test_bad_models_are_refused(tmp_path):
    config, w = util.model("mixed")
    folder = _folder(tmp_path, dict(config, architecture="Nobody"), w)
    with pytest.raises(ValueError, match="unknown architecture"):
        models.load_module(folder)
    short = dict(w)
    del short["l1.mix.right.lam"]
    with pytest.raises(KeyError, match="l1.mix.right.lam"):
        lovuzen.build(lovuzen.LovuzenConfig.from_dict(config), checkpoint.Weights.from_f32(short))
    wrong = dict(w, **{"l0.mlp.gate": w["l0.mlp.gate"][:-1]})
    with pytest.raises(ValueError, match="l0.mlp.gate"):
        lovuzen.build(lovuzen.LovuzenConfig.from_dict(config), checkpoint.Weights.from_f32(wrong))
    other = json.loads(json.dumps(config))
    other["layers"][0]["type"] = "serial"
    with pytest.raises(ValueError, match="serial"):
        lovuzen.LovuzenConfig.from_dict(other)


def test_bf16_host_tensors_round_to_nearest_even():
    t = ir.HostTensor.bf16(np.array([1.0, 1.00390625, 1.01171875, -2.5, 3.4e38], np.float32))
    assert t.numpy().tolist() == [1.0, 1.0, 1.015625, -2.5, math.inf]
    assert np.array_equal(ir.HostTensor.bf16(t.data.view(np.uint16)).numpy(), t.numpy())


def test_plain_implementation_reads_every_distance():
    """A key far away, and the first token, reach the last position's output through the reference's attention."""
    r = np.random.default_rng(3)
    T, H, G, d = 40, 4, 2, 8
    q, k = r.standard_normal((T, H, d)), r.standard_normal((T, G, d))
    bias = r.standard_normal((6, H))
    base = ref.attention(q, k, k, 0.3, bias, 20)
    for j in (0, 1, 38, 39):
        k2 = k.copy()
        k2[j] += 0.5
        moved = np.abs(ref.attention(q, k2, k2, 0.3, bias, 20) - base).max(axis=(1, 2))
        assert (moved[:j] == 0).all() and (moved[j:] > 1e-4).all()


def test_command_line_lists_models():
    r = subprocess.run([sys.executable, "-m", "onyxia_b200", "models"], cwd=ROOT, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=120)
    assert r.returncode == 0 and "Lovuzen" in r.stdout and "gemma3-1b-arch-int4" in r.stdout
