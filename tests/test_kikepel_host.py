"""Kikepel without a GPU: the configuration reader of the library, its refusals, and the oracle's mechanisms
against hand-checkable statements."""
from __future__ import annotations

import importlib
import json

import numpy as np
import pytest

import kikepel_oracle as oracle
from kikepel_util import artifacts, dense, latent, make_model, moe


@pytest.fixture(scope="module")
def rt(pkg):
    return importlib.import_module(f"{pkg.__name__}.runtime")


@pytest.fixture(scope="module")
def evo(pkg, rt):
    return rt.EvoLibrary(pkg.EVO_LIBRARY)


def test_configuration_comes_from_config_json(pkg, evo, tmp_path):
    layers = [latent(heads=7, mlp=dense(96)), latent(sink=False, mlp=moe(ff=130)), latent(mlp=None)]
    directory, _, _ = make_model(pkg, tmp_path / "m", layers, vocab=321, width=48, eps=3e-5)
    read, mixers = evo.read_model_config(directory)
    assert read.architecture == b"Kikepel" and mixers == [7, 7, 7]
    assert (read.vocab_size, read.width, read.layers, read.heads, read.inner_width) == (321, 48, 3, 7, 130)
    assert abs(read.epsilon - 3e-5) < 1e-10 and read.max_seqlen >= 1 << 20


def rewrite(directory, change):
    path = directory / "config.json"
    config = json.loads(path.read_text())
    change(config)
    path.write_text(json.dumps(config))


@pytest.mark.parametrize("change, code, text", [
    (lambda c: c["layers"][0].update(type="latent_attention_9"), 5, "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="maxout"), 5, "unknown kind"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), 4, "q_rank"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), 4, "size"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), 4, "mask"),
    (lambda c: c["layers"][0]["mixer"].update(dim=300), 5, "not supported"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=1100), 5, "not supported"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=80), 4, "unexpected dtype or shape"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), 4, "above the number of experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=2000), 5, "experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=9), 4, "unexpected dtype or shape"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), 4, "limit"),
    (lambda c: c["layers"][1].update(type="latent_attention"), 4, "sink"),
    (lambda c: c.pop("logit_scale"), 4, "logit_scale"),
    (lambda c: c.update(logit_softcap=0), 4, "logit_softcap"),
    (lambda c: c["norm"].pop("eps"), 4, "eps"),
    (lambda c: c.update(width=64), 4, "unexpected dtype or shape"),
    (lambda c: c.update(layers={}), 4, "layers"),
])
def test_inconsistent_configurations_are_refused(pkg, rt, evo, tmp_path, change, code, text):
    directory, _, _ = make_model(pkg, tmp_path / "m", [latent(mlp=dense()), latent(sink=False, mlp=moe())])
    rewrite(directory, change)
    with pytest.raises(rt.EvoError) as error:
        evo.read_model_config(directory)
    assert error.value.code == code and text in str(error.value)


def test_missing_expert_is_refused(pkg, rt, evo, tmp_path):
    _, config, weights = make_model(pkg, tmp_path / "m", [latent(mlp=moe(experts=3))])
    kept = {k: v.astype(np.float32) for k, v in weights.items() if k != "l0.mlp.e2.up"}
    artifacts(pkg).write_decoder(tmp_path / "missing", config, kept)
    with pytest.raises(rt.EvoError) as error:
        evo.read_model_config(tmp_path / "missing")
    assert error.value.code == 4 and "e2.up" in str(error.value)


def test_oracle_window_and_sink():
    assert list(oracle.visible_keys(9, 3)) == [7, 8, 9] and list(oracle.visible_keys(1, 3)) == [0, 1]
    assert np.allclose(oracle.softmax(np.array([0.0, 0.0]), np.log(2.0)), [0.25, 0.25])
    assert np.allclose(oracle.softmax(np.array([5.0]), None), [1.0])
    assert oracle.softmax(np.array([-700.0]), 2.0)[0] < 1e-200 and oracle.softmax(np.array([2.0]), -900.0)[0] == 1.0


def test_oracle_layer_norm_takes_the_mean_off():
    x = np.array([[1.0, 2.0, 3.0]]) + 100.0
    assert np.allclose(oracle.layer_norm(x, np.array([1.0, 1.0, 2.0]), 0.0), [[-1.22474487, 0.0, 2.44948974]])


def test_oracle_expert_clamps_and_weighs_its_input():
    one = np.ones((1, 1))
    y = oracle.expert(np.array([10.0]), one, -one, one, 2.0)           # g = 2, u = -2
    assert np.allclose(y, 2.0 * oracle.sigmoid(3.404) * -1.0)
    low = oracle.expert(np.array([-10.0]), one, one, one, 2.0)         # the gate is bounded from above only
    assert np.allclose(low, -10.0 * oracle.sigmoid(-17.02) * -1.0)
    mlp = moe(experts=2, top=2, ff=1, limit=50.0)
    w = {"router": np.array([[1.0], [-1.0]])} | {f"e{e}.{n}": one for e in range(2) for n in ("gate", "up", "down")}
    h = np.array([[0.7]])
    expected = sum(oracle.expert(s * h[0], one, one, one, 50.0) for s in oracle.sigmoid(np.array([0.7, -0.7])))
    assert np.allclose(oracle.mixture(h, w, "", mlp), expected)


def test_oracle_routes_to_the_largest_scores():
    chosen, weights = oracle.route(np.array([1.0]), np.array([[0.1], [3.0], [-1.0], [2.0]]), 3)
    assert list(chosen) == [1, 3, 0] and np.allclose(weights, oracle.sigmoid(np.array([3.0, 2.0, 0.1])))


def test_benchmark_work_counts_window_and_experts(pkg):
    bench = importlib.import_module(f"{pkg.__name__}.decoder_bench")
    art = artifacts(pkg)
    config = art.kikepel_config([latent(heads=2, dim=8, vdim=4, size=3, mlp=moe(experts=5, top=2, ff=16))], vocab=4, width=16)
    seen = sum(len(oracle.visible_keys(i, 3)) for i in range(10, 16))
    work = bench.latent_work(config, 6, 16)
    assert work["attention"][0] == 2.0 * 2 * 12 * seen and work["gemm_grouped"][0] == 6.0 * 12 * 16 * 16
    total = sum(2.0 * np.prod(s) for n, s in art.decoder_manifest(config) if ".e" not in n and n != "embed")
    assert bench.token_weight_bytes(config, art) == pytest.approx(total + 2.0 * 16 + 2 * 3 * 2.0 * 16 * 16)
