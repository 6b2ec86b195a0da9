"""Gigusun without a GPU: the configuration reader of the library, its refusals, and the oracle's mechanisms
against hand-checkable statements."""
from __future__ import annotations

import importlib
import json
import struct

import numpy as np
import pytest

import gigusun_oracle as oracle
from gigusun_util import artifacts, attention, delta, gla, make_model


@pytest.fixture(scope="module")
def rt(pkg):
    return importlib.import_module(f"{pkg.__name__}.runtime")


@pytest.fixture(scope="module")
def evo(pkg, rt):
    return rt.EvoLibrary(pkg.EVO_LIBRARY)


def test_configuration_comes_from_config_json(pkg, evo, tmp_path):
    layers = [delta(heads=6, kv_heads=3, dim=28), gla(dim=44), attention(heads=4, kv_heads=1, ff=None), gla(heads=5, ff=90)]
    directory, config, _ = make_model(pkg, tmp_path / "m", layers, vocab=321, width=48, max_positions=99, eps=3e-5)
    read, mixers = evo.read_model_config(directory)
    assert read.architecture == b"Gigusun" and mixers == [6, 5, 4, 5]
    assert (read.vocab_size, read.width, read.layers, read.max_seqlen) == (321, 48, 4, 99)
    assert (read.heads, read.inner_width, read.state_size, read.short_filter_length) == (6, 90, 44, 4)
    assert abs(read.epsilon - 3e-5) < 1e-10


def rewrite(directory, change):
    path = directory / "config.json"
    config = json.loads(path.read_text())
    change(config)
    path.write_text(json.dumps(config))


@pytest.mark.parametrize("change, code, text", [
    (lambda c: c.update(architecture="Unheard"), 5, "unknown architecture"),
    (lambda c: c["layers"][0].update(type="mamba"), 5, "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), 5, "dense"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), 4, "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("softcap"), 4, "softcap"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), 4, "size"),
    (lambda c: c["layers"][0]["mixer"].update(dim=27), 4, "unexpected dtype or shape"),
    (lambda c: c["layers"][0]["mixer"].update(dim=300), 5, "not supported"),
    (lambda c: c.update(width=64), 4, "unexpected dtype or shape"),
    (lambda c: c.update(vocab=1.5), 4, "integer"),
    (lambda c: c.pop("norm"), 4, "norm"),
    (lambda c: c.update(layers=[]), 4, "layers"),
])
def test_inconsistent_configurations_are_refused(pkg, rt, evo, tmp_path, change, code, text):
    directory, _, _ = make_model(pkg, tmp_path / "m", [delta(), attention()])
    rewrite(directory, change)
    with pytest.raises(rt.EvoError) as error:
        evo.read_model_config(directory)
    assert error.value.code == code and text in str(error.value)


def test_missing_tensors_are_refused_and_foreign_headers_are_read(pkg, rt, evo, tmp_path):
    directory, config, weights = make_model(pkg, tmp_path / "m", [gla()])
    art = artifacts(pkg)
    kept = {k: v.astype(np.float32) for k, v in weights.items() if k != "l0.mix.a2.b"}
    art.write_decoder(tmp_path / "missing", config, kept)
    with pytest.raises(rt.EvoError) as error:
        evo.read_model_config(tmp_path / "missing")
    assert error.value.code == 4 and "a2.b" in str(error.value)
    # an unpadded header and an integer tensor that the design does not use
    raw = (directory / "model.safetensors").read_bytes()
    length = struct.unpack("<Q", raw[:8])[0]
    header = json.loads(raw[8:8 + length])
    header.pop("__metadata__")
    payload = raw[8 + length:] + b"\0" * 8
    header["table"] = {"dtype": "I32", "shape": [2], "data_offsets": [len(payload) - 8, len(payload)]}
    text = json.dumps(header).encode()
    text += b" " * ((3 - len(text)) % 8)
    assert len(text) % 8 != 0
    (directory / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + payload)
    assert evo.read_model_config(directory)[0].layers == 1


def test_oracle_window_keeps_the_first_tokens():
    assert list(oracle.visible_keys(9, 3, 2)) == [0, 1, 7, 8, 9]
    assert list(oracle.visible_keys(2, 5, 1)) == [0, 1, 2]
    assert list(oracle.visible_keys(4, 4, 0)) == [1, 2, 3, 4]


def test_oracle_sink_takes_its_share():
    assert np.allclose(oracle.softmax_with_sink(np.array([0.0])), [0.5])
    assert np.allclose(oracle.softmax_with_sink(np.array([800.0, 800.0])), [0.5, 0.5])
    assert oracle.softmax_with_sink(np.array([-700.0]))[0] < 1e-200


def test_oracle_delta_rule_replaces_what_a_key_holds():
    """With beta = 1 and no decay a repeated unit key reads back its latest value."""
    rng = np.random.default_rng(0)
    key = np.zeros((3, 1, 4))
    key[:, 0, 1] = 1.0
    values = rng.normal(size=(3, 1, 5))
    out, state = oracle.gated_delta_rule(key, key, values, np.ones((3, 1)), np.ones((3, 1)))
    assert np.allclose(out, values) and np.allclose(state[0, 1], values[2, 0])


def test_oracle_linear_attention_carries_its_state():
    rng = np.random.default_rng(1)
    q, k, v = (rng.normal(size=(11, 2, n)) for n in (3, 3, 4))
    a = rng.uniform(0.2, 1.0, (11, 2, 3))
    whole, state = oracle.gated_linear_attention(q, k, v, a)
    head, middle = oracle.gated_linear_attention(q[:5], k[:5], v[:5], a[:5])
    tail, end = oracle.gated_linear_attention(q[5:], k[5:], v[5:], a[5:], middle)
    assert np.allclose(np.concatenate([head, tail]), whole) and np.allclose(end, state)


def test_oracle_convolution_meets_the_current_token_last():
    x = np.arange(1.0, 5.0)[:, None]
    assert np.allclose(oracle.causal_convolution(x, np.array([[100.0, 10.0, 1.0]]))[:, 0], [1, 12, 123, 234])


def test_benchmark_work_counts_the_window(pkg):
    bench = importlib.import_module(f"{pkg.__name__}.decoder_bench")
    art = artifacts(pkg)
    config = art.gigusun_config([attention(heads=2, kv_heads=1, dim=8, vdim=8, size=3, keep_first=2)], vocab=4, width=16,
                                max_positions=64)
    seen = sum(len(oracle.visible_keys(i, 3, 2)) for i in range(10, 16))
    assert bench.class_work(config, 6, 16)["attention"][0] == 2.0 * 2 * 16 * seen
