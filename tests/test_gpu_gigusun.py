"""Gigusun models through the runtime: whole prompts, portions, decoding, reuse of contexts, scheduling, greedy
generation, the command line and trace replay, against the float64 oracle and against each other."""
from __future__ import annotations

import importlib
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

import gigusun_oracle as oracle
from gigusun_util import attention, delta, gla, make_model

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
LAYERS = [delta(), attention(), gla(), delta(heads=3, kv_heads=3, dim=12, vdim=44, conv=2, ff=None),
          attention(heads=4, kv_heads=4, dim=72, vdim=64, size=70, keep_first=0, softcap=9.0, ff=136), gla(heads=2, dim=64, vdim=16)]
SHARP = 3.0


def sharpen(weights):
    """Query norms scaled up, so that single keys stand out of the softmax."""
    for name in weights:
        if name.endswith("q.norm"):
            weights[name] *= SHARP


@pytest.fixture(scope="module")
def rt(pkg):
    import torch

    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    return importlib.import_module(f"{pkg.__name__}.runtime")


@pytest.fixture(scope="module")
def made(pkg, rt, tmp_path_factory):
    directory, config, weights = make_model(pkg, tmp_path_factory.mktemp("gigusun") / "m", LAYERS, edit=sharpen)
    tokens = np.random.default_rng(11).integers(0, config["vocab"], 230).tolist()
    residuals: list = []
    logits = oracle.forward(config, weights, tokens, residuals)
    evo = rt.EvoLibrary(pkg.EVO_LIBRARY)
    return dict(directory=directory, config=config, weights=weights, tokens=tokens, logits=logits, residuals=residuals,
                evo=evo, model=evo.load(directory))


def error(actual, expected):
    """Largest per-row root-mean-square difference of logits, in units of the logits' own spread."""
    d = np.asarray(actual, np.float64) - expected
    d = d - d.mean(axis=-1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=-1)).max() / expected.std())


F32_LIMIT, BF16_LIMIT = 1e-4, 8e-2
PROFILES = pytest.mark.parametrize("profile, limit", [("float32", F32_LIMIT), ("exact", BF16_LIMIT)])


def context(rt, made, profile, size=256):
    return made["model"].context(size, flags=rt.CONTEXT_FLAG_FLOAT32 if profile == "float32" else 0)


@PROFILES
def test_whole_prompt_and_residual_stream(rt, made, profile, limit):
    c = context(rt, made, profile)
    assert c.profile == profile and made["model"].vocab == 300 and made["model"].layers == 6
    assert error(c.prefill_tokens(made["tokens"]), made["logits"]) < limit
    for layer, expected in enumerate(made["residuals"]):
        got = c.embed_tokens(made["tokens"], layer)
        assert error(got, expected) < limit, layer
    c.close()


@PROFILES
def test_token_by_token_equals_the_prompt(rt, made, profile, limit):
    """Decoding from the first token on, past every window, through the captured step."""
    c = context(rt, made, profile)
    rows = [c.prefill_tokens(made["tokens"][:1])[0]] + [c.decode(t) for t in made["tokens"][1:]]
    assert error(np.array(rows), made["logits"]) < limit
    assert c.position == len(made["tokens"])
    c.close()


@PROFILES
@pytest.mark.parametrize("portions", [[2] * 115, [1, 2, 3] * 38 + [2], [13, 70, 1, 96, 50], [128, 2, 100], [229, 1], [8, 9, 33, 180]])
def test_portions(rt, made, profile, limit, portions):
    c = context(rt, made, profile)
    got, at = [], 0
    for n in portions:
        part = made["tokens"][at:at + n]
        if at == 0:
            got.append(c.prefill_tokens(part))
        elif n == 1:
            got.append(c.decode(part[0])[None])
        else:
            got.append(c.prefill_tokens(part, c.PREFILL_CHUNK))
        at += n
    assert at == len(made["tokens"])
    assert error(np.concatenate(got), made["logits"]) < limit
    c.close()


@PROFILES
def test_contexts_are_used_again(rt, made, profile, limit):
    """A context that held another sequence gives the same logits as a new one, also after a longer sequence."""
    c = context(rt, made, profile)
    other = np.random.default_rng(5).integers(0, 300, 250).tolist()
    for _ in range(2):
        c.prefill_tokens(other)
        c.decode(7)
        first = c.prefill_tokens(made["tokens"][:100])
        rest = np.array([c.decode(t) for t in made["tokens"][100:140]])
        assert error(np.concatenate([first, rest]), made["logits"][:140]) < limit
    stateless = c.prefill_tokens(made["tokens"], c.PREFILL_STATELESS)
    assert error(stateless, made["logits"]) < limit and c.position == 0
    cached = c.prefill_tokens(made["tokens"][:60], c.PREFILL_CACHED)
    more = c.prefill_tokens(made["tokens"][60:90], c.PREFILL_CHUNK)
    assert error(np.concatenate([cached, more]), made["logits"][:90]) < limit
    c.close()


def test_values_that_are_one(pkg, rt, tmp_path):
    """One head, one channel group, one tap, a window of one, no feed-forward, a vocabulary below a tile."""
    layers = [delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, ff=None), attention(heads=1, kv_heads=1, dim=8, vdim=8, size=1,
              keep_first=1, ff=None), gla(heads=1, dim=1, vdim=1, tau=1.0, ff=8), attention(heads=2, kv_heads=1, dim=1, vdim=3,
              size=300, keep_first=40)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=19, width=24, max_positions=90, decay_rank=1)
    tokens = np.random.default_rng(2).integers(0, 19, 80).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = rt.EvoLibrary(pkg.EVO_LIBRARY).load(directory)
    for flags, limit in ((rt.CONTEXT_FLAG_FLOAT32, F32_LIMIT * 5), (0, 0.15)):
        c = model.context(90, flags=flags)
        assert error(c.prefill_tokens(tokens), expected) < limit
        rows = [c.prefill_tokens(tokens[:3])] + [c.decode(t)[None] for t in tokens[3:]]
        assert error(np.concatenate(rows), expected) < limit
        c.close()
    with pytest.raises(rt.EvoError):
        model.context(91)                                           # beyond the learned positions
    model.close()


def test_odd_sizes_everywhere(pkg, rt, tmp_path):
    """No width is a multiple of eight: the scalar forms of every operator, rows of every kernel's range."""
    layers = [attention(heads=5, kv_heads=5, dim=33, vdim=7, size=19, keep_first=2, ff=37), delta(heads=3, kv_heads=1, dim=65, vdim=9,
              conv=9, ff=None), gla(heads=3, dim=130, vdim=11, tau=0.7, ff=51), delta(heads=2, kv_heads=2, dim=7, vdim=70, conv=5, ff=29)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=101, width=51, max_positions=163, eps=1e-3,
                                            decay_rank=9, edit=sharpen)
    tokens = np.random.default_rng(9).integers(0, 101, 163).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = rt.EvoLibrary(pkg.EVO_LIBRARY).load(directory)
    for flags, limit in ((rt.CONTEXT_FLAG_FLOAT32, F32_LIMIT), (0, BF16_LIMIT)):
        c = model.context(163, flags=flags)
        assert error(c.prefill_tokens(tokens), expected) < limit
        got, at = [], 0
        for n in (3, 40, 1, 12, 2, 64, 1, 40):
            got.append(c.prefill_tokens(tokens[:n]) if at == 0 else c.decode(tokens[at])[None] if n == 1
                       else c.prefill_tokens(tokens[at:at + n], c.PREFILL_CHUNK))
            at += n
        assert at == 163 and error(np.concatenate(got), expected) < limit
        c.close()
    model.close()


def test_larger_heads_on_the_tensor_cores(pkg, rt, tmp_path):
    layers = [attention(heads=4, kv_heads=2, dim=128, vdim=96, size=100, keep_first=5, ff=320), delta(heads=4, kv_heads=2, dim=128,
              vdim=64, ff=512), gla(heads=2, dim=128, vdim=128, ff=None)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=640, width=256, max_positions=700, edit=sharpen)
    tokens = np.random.default_rng(8).integers(0, 640, 420).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = rt.EvoLibrary(pkg.EVO_LIBRARY).load(directory)
    for flags, limit in ((rt.CONTEXT_FLAG_FLOAT32, F32_LIMIT), (0, BF16_LIMIT)):
        c = model.context(500, flags=flags)
        assert error(c.prefill_tokens(tokens), expected) < limit
        rows = [c.prefill_tokens(tokens[:200]), c.prefill_tokens(tokens[200:333], c.PREFILL_CHUNK),
                c.prefill_tokens(tokens[333:335], c.PREFILL_CHUNK)] + [c.decode(t)[None] for t in tokens[335:]]
        assert error(np.concatenate(rows), expected) < limit
        c.close()
    model.close()


def test_prompt_longer_than_the_activation_arena(pkg, rt, tmp_path):
    """Chunks of the arena size against one pass of the same tokens in smaller portions."""
    layers = [attention(heads=2, kv_heads=1, dim=64, vdim=64, size=200, keep_first=2, ff=None), delta(ff=None), gla(ff=None)]
    directory, _, _ = make_model(pkg, tmp_path / "m", layers, width=64, max_positions=9000)
    model = rt.EvoLibrary(pkg.EVO_LIBRARY).load(directory)
    tokens = np.random.default_rng(4).integers(0, 300, 8700).tolist()
    c = model.context(9000)
    assert c.activation_capacity == 8192
    whole = c.prefill_tokens(tokens)
    parts = [c.prefill_tokens(tokens[:5000]), c.prefill_tokens(tokens[5000:], c.PREFILL_CHUNK)]
    assert error(np.concatenate(parts), whole.astype(np.float64)) < BF16_LIMIT
    c.close()
    model.close()


def greedy(logits_of, prompt, count):
    row, out = logits_of(prompt), []
    for i in range(count):
        out.append(int(row.argmax()))
        if i + 1 < count:
            row = logits_of([out[-1]])
    return out


def test_greedy_generation_through_the_scheduler(rt, made):
    """Unequal requests on a pool of contexts: the same ids as one context alone, which are the oracle's."""
    rng = np.random.default_rng(21)
    prompts = [rng.integers(0, 300, n).tolist() for n in (1, 3, 40, 90, 17, 2, 150, 64)]
    pool = rt.Scheduler(made["model"], workers=3, maximum_queue=32, context_size=200, flags=rt.CONTEXT_FLAG_FLOAT32)
    tickets = [pool.generate_tokens(p, 6) for p in prompts]
    score = pool.score_tokens(made["tokens"][:120])
    sampled = pool.generate_tokens(prompts[3], 5, temperature=0.9, top_k=7, seed=3)
    too_long = pool.generate_tokens(prompts[6], 60)
    outside = pool.generate_tokens([5, 300], 2)
    pool.wait_idle()
    for prompt, ticket in zip(prompts, tickets):
        result = pool.results[ticket]
        assert result["status"] == 0, result
        c = context(rt, made, "float32")
        alone = greedy(lambda ids: c.prefill_tokens(ids)[-1] if c.position == 0 else c.decode(ids[0]), prompt, 6)
        c.close()
        assert result["generated_tokens"] == alone and result["generated"] == b""
        sequence = list(prompt)
        for token in alone[:3]:
            row = oracle.forward(made["config"], made["weights"], sequence)[-1]
            assert row.max() - row[token] < 1e-3 * row.std()
            sequence.append(token)
    lp = made["logits"][:120] - np.logaddexp.reduce(made["logits"][:120], axis=1)[:, None]
    expected = float(sum(lp[i, made["tokens"][i + 1]] for i in range(119)))
    assert abs(pool.results[score]["log_likelihood"] - expected) < 1e-2
    assert len(pool.results[sampled]["generated_tokens"]) == 5
    assert pool.results[too_long]["status"] == 2 and pool.results[outside]["status"] == 2
    late = pool.generate_tokens(prompts[2], 6)                       # the worker whose request failed still serves
    pool.wait_idle()
    assert pool.results[late]["generated_tokens"] == pool.results[tickets[2]]["generated_tokens"]
    pool.close()


def cli(*arguments, stdin=""):
    return subprocess.run([str(ROOT / "evo.cpp_b200" / "evo"), *map(str, arguments)], input=stdin, capture_output=True, text=True,
                          timeout=120)


def test_command_line(rt, made):
    prompt = made["tokens"][:30]
    c = context(rt, made, "float32")
    expected = greedy(lambda ids: c.prefill_tokens(ids)[-1] if c.position == 0 else c.decode(ids[0]), prompt, 8)
    c.close()
    ids = ",".join(map(str, prompt))
    run = cli("run", "-m", made["directory"], "--prompt-tokens", ids, "-n", 8, "--ctx", 64, "--profile", "float32")
    assert run.returncode == 0, run.stderr
    assert [int(t) for t in run.stdout.split(",")] == expected
    forced = cli("run", "-m", made["directory"], "--prompt-tokens", ids, "-n", 8, "--ctx", 64, "--profile", "float32",
                 "--force-prompt-threshold", 11)
    assert forced.stdout == run.stdout
    requests = [{"id": "g", "op": "generate", "prompt_tokens": prompt, "tokens": 8}, {"id": "s", "op": "score", "tokens": prompt}]
    serve = cli("serve", "-m", made["directory"], "--ctx", 64, "--profile", "float32", "--workers", 2,
                stdin="".join(json.dumps(r) + "\n" for r in requests))
    answers = {a["id"]: a for a in map(json.loads, serve.stdout.splitlines())}
    assert answers["g"]["generated_tokens"] == expected and answers["s"]["scored_tokens"] == 29
    assert cli("run", "-m", made["directory"], "--prompt-tokens", "1,x", "-n", 1).returncode == 2
    assert cli("run", "-m", made["directory"], "--prompt-tokens", "1,2", "-n", 1, "--profile", "b200-fp8", "--ctx", 64).returncode == 5


def replay(directory, dtype, out, steps, model=None):
    out.mkdir()
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(model or directory), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "400"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                         timeout=600)
    return run


@pytest.mark.parametrize("dtype, limit", [("float32", F32_LIMIT), ("bfloat16", BF16_LIMIT)])
def test_trace_replay(made, tmp_path, dtype, limit):
    t = made["tokens"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[50:52], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": t[:20], "want": [19]}, {"id": "a", "tokens": [t[52]], "want": [0]}], "end": ["b"]},
             {"step": 7, "entries": [{"id": "c", "tokens": t[:9], "want": [0, 8]}, {"id": "a", "tokens": t[53:90], "want": [36]}],
              "end": ["a", "c"]}]
    run = replay(made["directory"], dtype, tmp_path / "out", steps)
    assert run.returncode == 0, run.stderr
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    assert sorted(p.name for p in (tmp_path / "out").iterdir()) == ["0.f32", "2.f32", "7.f32"]
    for name, places in (("0", [49, 3]), ("2", [19, 52]), ("7", [0, 8, 89])):
        got = np.fromfile(tmp_path / "out" / f"{name}.f32", np.float32).reshape(len(places), -1)
        assert error(got, made["logits"][places]) < limit


def test_trace_replay_refusals(made, tmp_path):
    tiny = ROOT / "tests" / "golden" / "tiny" / "tiny.safetensors"
    bad = replay(made["directory"], "float32", tmp_path / "a", [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": [2]}]}])
    assert bad.returncode == 2 and "wants a place outside" in bad.stderr
    refused = subprocess.run([str(ROOT / "evo.cpp_b200" / "evo"), "replay", "-m", str(tiny), "--allow-test-fixture", "--dtype", "float32",
                              "--out", str(tmp_path), "--max-tokens", "16"], input="", capture_output=True, text=True, timeout=120)
    assert refused.returncode == 3


def test_taps(rt, made):
    c = context(rt, made, "float32")
    logits, taps = c.prefill_with_dumps(bytes([1, 2, 3, 250]), [(1, "block_output"), (1, "mixer_output"), (2, "pre_norm"), (2, "mlp_activation")])
    expected: list = []
    full = oracle.forward(made["config"], made["weights"], [1, 2, 3, 250], expected)
    assert error(logits, full) < F32_LIMIT and error(taps[(1, "block_output")], expected[1]) < F32_LIMIT
    eps = made["config"]["norm"]["eps"]
    assert error(taps[(2, "pre_norm")], oracle.centred_rms_norm(expected[1], made["weights"]["l2.norm1"], eps)) < F32_LIMIT
    assert taps[(1, "mixer_output")].shape == (4, 6 * 24) and taps[(2, "mlp_activation")].shape == (4, 72)
    with pytest.raises(rt.EvoError) as refused:
        c.prefill_with_dumps(b"ab", [(1, "mixer_filter")])
    assert refused.value.code == 5
    c.close()


def test_refusals(rt, made):
    model = made["model"]
    for flags in (rt.CONTEXT_FLAG_FAST_Q8_KV, rt.CONTEXT_FLAG_FP8_FFN):
        with pytest.raises(rt.EvoError) as refused:
            model.context(64, flags=flags)
        assert refused.value.code == 5
    with pytest.raises(rt.EvoError) as refused:
        made["evo"].load_slice(made["directory"], 0, 0, 2)
    assert refused.value.code == 5
    c = model.context(8)
    with pytest.raises(rt.EvoError):
        c.prefill_tokens(list(range(9)))
    c.prefill_tokens([1, 2, 3])
    with pytest.raises(rt.EvoError):
        c.prefill_tokens([1] * 6, c.PREFILL_CHUNK)
    c.close()
    c = model.context(8)
    c.prefill_tokens([1] * 8)
    with pytest.raises(rt.EvoError):
        c.decode(1)                                                 # the context is full
    c.close()
