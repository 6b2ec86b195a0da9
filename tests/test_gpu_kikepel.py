"""Kikepel models through the runtime: whole prompts, portions, decoding, reuse of contexts, scheduling, greedy
generation, the command line and trace replay, against the float64 oracle and against each other."""
from __future__ import annotations

import importlib
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

import kikepel_oracle as oracle
from kikepel_util import dense, latent, make_model, moe

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
LAYERS = [latent(mlp=moe()),
          latent(heads=3, dim=64, vdim=64, q_rank=32, kv_rank=48, size=70, sink=False, mlp=dense()),
          latent(heads=8, dim=16, vdim=8, q_rank=24, kv_rank=136, size=9, scale=0.4, mlp=None),
          latent(heads=2, dim=72, vdim=128, q_rank=72, kv_rank=264, size=130, mlp=moe(experts=3, top=1, ff=136, limit=2.5)),
          latent(heads=4, dim=40, vdim=24, q_rank=80, kv_rank=64, size=1, sink=False, mlp=moe(experts=5, top=5, ff=24, limit=0.3))]
SHARP = 3.0


def sharpen(weights):
    """Query latents scaled up, so that single keys stand out of the softmax."""
    for name in weights:
        if name.endswith("dq.norm"):
            weights[name] *= SHARP


@pytest.fixture(scope="module")
def rt(pkg):
    import torch

    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    return importlib.import_module(f"{pkg.__name__}.runtime")


@pytest.fixture(scope="module")
def evo(pkg, rt):
    return rt.EvoLibrary(pkg.EVO_LIBRARY)


def make_case(pkg, evo, directory, edit):
    directory, config, weights = make_model(pkg, directory, LAYERS, edit=edit)
    tokens = np.random.default_rng(11).integers(0, config["vocab"], 230).tolist()
    residuals: list = []
    logits = oracle.forward(config, weights, tokens, residuals)
    return dict(directory=directory, config=config, weights=weights, tokens=tokens, logits=logits, residuals=residuals,
                evo=evo, model=evo.load(directory))


@pytest.fixture(scope="module")
def made(pkg, evo, tmp_path_factory):
    return make_case(pkg, evo, tmp_path_factory.mktemp("kikepel") / "m", sharpen)


@pytest.fixture(scope="module")
def cases(pkg, evo, made, tmp_path_factory):
    """By profile.  The BF16 one is not sharpened: a token that takes another expert because two scores are nearly
    equal would move every row whose softmax has settled on that token."""
    return {"float32": made, "exact": make_case(pkg, evo, tmp_path_factory.mktemp("kikepel") / "plain", None)}


def row_errors(actual, expected):
    """Root-mean-square difference of every row, mean taken off, in units of the expected values' spread."""
    d = np.asarray(actual, np.float64) - expected
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / expected.std()


F32_LIMIT, BF16_LIMIT = 1e-4, 8e-2
PROFILES = pytest.mark.parametrize("profile", ["float32", "exact"])


def assert_close(actual, expected, profile, experts=True):
    """F32: every row.  BF16: every row, but with experts a twentieth of the rows may have taken another expert than
    the oracle where two scores are nearly equal."""
    e = row_errors(actual, expected)
    assert np.isfinite(e).all()
    if profile == "float32":
        assert e.max() < F32_LIMIT, e.max()
    else:
        assert (e > BF16_LIMIT).mean() <= (0.05 if experts else 0.0), np.sort(e)[-8:]


def context(rt, model, profile, size=256):
    return model.context(size, flags=rt.CONTEXT_FLAG_FLOAT32 if profile == "float32" else 0)


def in_portions(c, tokens, portions):
    got, at = [], 0
    for n in portions:
        part = tokens[at:at + n]
        if at == 0:
            got.append(c.prefill_tokens(part))
        elif n == 1:
            got.append(c.decode(part[0])[None])
        else:
            got.append(c.prefill_tokens(part, c.PREFILL_CHUNK))
        at += n
    assert at == len(tokens)
    return np.concatenate(got)


@PROFILES
def test_whole_prompt_and_residual_stream(rt, cases, profile):
    made = cases[profile]
    c = context(rt, made["model"], profile)
    assert c.profile == profile and made["model"].vocab == 300 and made["model"].layers == 5
    assert_close(c.prefill_tokens(made["tokens"]), made["logits"], profile)
    for layer, expected in enumerate(made["residuals"]):
        assert_close(c.embed_tokens(made["tokens"], layer), expected, profile)
    c.close()


@PROFILES
def test_token_by_token_equals_the_prompt(rt, cases, profile):
    """Decoding from the first token on, past every window, through the captured step."""
    made = cases[profile]
    c = context(rt, made["model"], profile)
    assert_close(in_portions(c, made["tokens"], [1] * 230), made["logits"], profile)
    assert c.position == 230
    c.close()


@PROFILES
@pytest.mark.parametrize("portions", [[2] * 115, [1, 2, 3] * 38 + [2], [13, 70, 1, 96, 50], [128, 2, 100], [229, 1], [8, 9, 33, 180]])
def test_portions(rt, cases, profile, portions):
    made = cases[profile]
    c = context(rt, made["model"], profile)
    assert_close(in_portions(c, made["tokens"], portions), made["logits"], profile)
    c.close()


@PROFILES
def test_contexts_are_used_again(rt, cases, profile):
    """A context that held another sequence gives the same logits as a new one, also after a longer sequence."""
    made = cases[profile]
    c = context(rt, made["model"], profile)
    other = np.random.default_rng(5).integers(0, 300, 250).tolist()
    for _ in range(2):
        c.prefill_tokens(other)
        c.decode(7)
        first = c.prefill_tokens(made["tokens"][:100])
        rest = np.array([c.decode(t) for t in made["tokens"][100:140]])
        assert_close(np.concatenate([first, rest]), made["logits"][:140], profile)
    assert_close(c.prefill_tokens(made["tokens"], c.PREFILL_STATELESS), made["logits"], profile)
    assert c.position == 0
    cached = c.prefill_tokens(made["tokens"][:60], c.PREFILL_CACHED)
    more = c.prefill_tokens(made["tokens"][60:90], c.PREFILL_CHUNK)
    assert_close(np.concatenate([cached, more]), made["logits"][:90], profile)
    c.close()


def test_values_that_are_one(pkg, rt, evo, tmp_path):
    """One head, one dimension, ranks of one, one expert, a window of one, a vocabulary below a tile."""
    layers = [latent(heads=1, dim=8, vdim=8, q_rank=8, kv_rank=8, size=1, mlp=moe(experts=1, top=1, ff=1, limit=1.0)),
              latent(heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, size=5, scale=1.0, sink=False, mlp=dense(1)),
              latent(heads=2, dim=1, vdim=3, q_rank=2, kv_rank=1, size=300, mlp=None)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=19, width=24, logit_scale=1.0, logit_softcap=1.0)
    tokens = np.random.default_rng(2).integers(0, 19, 80).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = evo.load(directory)
    c = context(rt, model, "float32", 90)
    assert row_errors(c.prefill_tokens(tokens), expected).max() < 1e-3
    assert row_errors(in_portions(c, tokens, [3] + [1] * 77), expected).max() < 1e-3
    c.close()
    c = context(rt, model, "exact", 90)
    whole = c.prefill_tokens(tokens)                                 # (norms of single values amplify BF16 rounding)
    assert np.isfinite(whole).all() and np.median(row_errors(whole, expected)) < 0.2
    c.close()
    model.close()


def test_odd_sizes_everywhere(pkg, rt, evo, tmp_path):
    """No width is a multiple of eight: the scalar forms of every operator, rows of every kernel's range."""
    layers = [latent(heads=5, dim=33, vdim=7, q_rank=19, kv_rank=45, size=19, mlp=moe(experts=7, top=3, ff=37)),
              latent(heads=3, dim=65, vdim=9, q_rank=77, kv_rank=301, size=150, sink=False, mlp=dense(51)),
              latent(heads=1, dim=130, vdim=201, q_rank=5, kv_rank=9, size=40, mlp=None)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=101, width=51, eps=1e-3)
    tokens = np.random.default_rng(9).integers(0, 101, 163).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = evo.load(directory)
    for profile in ("float32", "exact"):
        c = context(rt, model, profile, 163)
        assert_close(c.prefill_tokens(tokens), expected, profile)
        assert_close(in_portions(c, tokens, (3, 40, 1, 12, 2, 64, 1, 40)), expected, profile)
        c.close()
    model.close()


@pytest.mark.parametrize("mlp", [dense(320), moe(experts=4, top=2, ff=192, limit=1.5)], ids=["dense", "experts"])
def test_larger_heads_on_the_tensor_cores(pkg, rt, evo, tmp_path, mlp):
    layers = [latent(heads=4, dim=128, vdim=96, q_rank=192, kv_rank=256, size=100, mlp=mlp),
              latent(heads=2, dim=64, vdim=128, q_rank=64, kv_rank=512, size=333, sink=False, mlp=mlp)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, vocab=640, width=256, edit=sharpen)
    tokens = np.random.default_rng(8).integers(0, 640, 420).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = evo.load(directory)
    for profile in ("float32", "exact"):
        c = context(rt, model, profile, 500)
        assert_close(c.prefill_tokens(tokens), expected, profile, experts=mlp["kind"] == "moe")
        assert_close(in_portions(c, tokens, [200, 133, 2] + [1] * 85), expected, profile, experts=mlp["kind"] == "moe")
        c.close()
    model.close()


def test_many_rows_per_expert(pkg, rt, evo, tmp_path):
    """Prompts long enough for row tiles of CTA pairs, against the same tokens in smaller portions and the oracle."""
    layers = [latent(heads=2, dim=64, vdim=64, q_rank=64, kv_rank=64, size=30, mlp=moe(experts=2, top=2, ff=128, limit=1.0)),
              latent(heads=2, dim=64, vdim=64, q_rank=64, kv_rank=64, size=64, sink=False, mlp=moe(experts=2, top=1, ff=256, limit=4.0))]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, width=256)
    tokens = np.random.default_rng(3).integers(0, 300, 1300).tolist()
    expected = oracle.forward(config, weights, tokens)
    model = evo.load(directory)
    for profile in ("float32", "exact"):
        c = context(rt, model, profile, 1300)
        assert_close(c.prefill_tokens(tokens), expected, profile)
        assert_close(in_portions(c, tokens, [400, 17, 883]), expected, profile)
        c.close()
    model.close()


def test_far_edges_of_windows_in_prompts_and_decoding(pkg, rt, evo, tmp_path):
    """A sequence of one common token with a single rare one: with scores that make the rare token's key stand out, the
    logits of every later position tell whether it was still in the window."""
    size = 37
    layers = [latent(heads=4, dim=64, vdim=64, q_rank=96, kv_rank=64, size=size, sink=False, scale=2.0, mlp=None)]
    directory, config, weights = make_model(pkg, tmp_path / "m", layers, edit=sharpen)
    tokens = [5] * 120
    tokens[30] = 211
    expected = oracle.forward(config, weights, tokens)
    baseline = oracle.forward(config, weights, [5] * 120)
    change = np.abs(expected - baseline).max(axis=1)
    assert change[30 + size - 1] > 1e-2 and change[30 + size:].max() < 1e-12          # the window's edge shows
    model = evo.load(directory)
    for profile in ("float32", "exact"):
        c = context(rt, model, profile, 120)
        for portions in ([120], [1] * 120, [31, 35, 1, 1, 1, 51], [64, 2, 2, 2, 50], [20, 9, 38, 53]):
            got = in_portions(c, tokens, portions)
            assert_close(got, expected, profile, experts=False)
            # rows on the two sides of the edge differ by what the rare token adds
            outside = got[30 + size:]
            assert np.abs(outside - outside[-1]).max() < (1e-4 if profile == "float32" else 0.25) * max(change[30 + size - 1], 1e-2) * 4
        c.close()
    model.close()


def test_prompt_longer_than_the_activation_arena(pkg, rt, evo, tmp_path):
    """Chunks of the arena size against one pass of the same tokens in smaller portions."""
    layers = [latent(heads=2, dim=64, vdim=64, q_rank=64, kv_rank=64, size=200, mlp=dense(64)),
              latent(heads=1, dim=64, vdim=64, q_rank=64, kv_rank=64, size=5000, sink=False, mlp=None)]
    directory, _, _ = make_model(pkg, tmp_path / "m", layers, width=64)
    model = evo.load(directory)
    tokens = np.random.default_rng(4).integers(0, 300, 8700).tolist()
    c = model.context(9000)
    assert c.activation_capacity == 8192
    whole = c.prefill_tokens(tokens)
    parts = np.concatenate([c.prefill_tokens(tokens[:5000]), c.prefill_tokens(tokens[5000:], c.PREFILL_CHUNK)])
    assert row_errors(parts, whole.astype(np.float64)).max() < BF16_LIMIT
    c.close()
    model.close()


def greedy(c, prompt, count):
    row, out = c.prefill_tokens(prompt)[-1], []
    for i in range(count):
        out.append(int(row.argmax()))
        if i + 1 < count:
            row = c.decode(out[-1])
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
        c = context(rt, made["model"], "float32")
        alone = greedy(c, prompt, 6)
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


def test_long_decoding(pkg, rt, evo, tmp_path):
    """Generation many windows long, replayed as one prompt."""
    layers = [latent(heads=4, dim=32, vdim=48, q_rank=48, kv_rank=64, size=25, mlp=dense(64)),
              latent(heads=2, dim=48, vdim=32, q_rank=64, kv_rank=32, size=90, sink=False, mlp=moe(experts=4, top=2, ff=48, limit=1.0))]
    directory, _, _ = make_model(pkg, tmp_path / "m", layers, edit=sharpen)
    model = evo.load(directory)
    c = context(rt, model, "float32", 700)
    rows = [c.prefill_tokens([3, 1, 4])[-1]]
    sequence = [3, 1, 4]
    rng = np.random.default_rng(6)
    for _ in range(600):
        best = np.argsort(-rows[-1])[:5]
        sequence.append(int(best[rng.integers(5)]))                   # (greedy ids alone would soon repeat)
        rows.append(c.decode(sequence[-1]))
    whole = c.prefill_tokens(sequence)
    assert row_errors(np.array(rows), whole[2:].astype(np.float64)).max() < F32_LIMIT
    c.close()
    model.close()


def cli(*arguments, stdin=""):
    return subprocess.run([str(ROOT / "evo.cpp_b200" / "evo"), *map(str, arguments)], input=stdin, capture_output=True, text=True,
                          timeout=120)


def test_command_line(rt, made):
    prompt = made["tokens"][:30]
    c = context(rt, made["model"], "float32")
    expected = greedy(c, prompt, 8)
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
    assert cli("run", "-m", made["directory"], "--prompt-tokens", "1,2", "-n", 1, "--profile", "b200-fp8", "--ctx", 64).returncode == 5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(cases, tmp_path, dtype):
    made = cases["float32" if dtype == "float32" else "exact"]
    t = made["tokens"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[50:52], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": t[:20], "want": [19]}, {"id": "a", "tokens": [t[52]], "want": [0]}], "end": ["b"]},
             {"step": 7, "entries": [{"id": "c", "tokens": t[:9], "want": list(range(9))}, {"id": "a", "tokens": t[53:90], "want": [36]}],
              "end": ["a", "c"]}]
    (tmp_path / "out").mkdir()
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(made["directory"]), "--dtype", dtype, "--out",
                          str(tmp_path / "out"), "--max-tokens", "400"], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    got = np.concatenate([np.fromfile(tmp_path / "out" / f"{name}.f32", np.float32).reshape(-1, 300) for name in (0, 2, 7)])
    e = row_errors(got, made["logits"][[49, 3, 19, 52, *range(9), 89]])
    assert e.max() < F32_LIMIT if dtype == "float32" else (e > BF16_LIMIT).sum() <= 1, e


def test_taps(rt, made):
    c = context(rt, made["model"], "float32")
    points = [(1, "block_output"), (1, "mixer_output"), (1, "mixer_projection"), (3, "mixer_residual")]
    logits, taps = c.prefill_with_dumps(bytes([1, 2, 3, 250]), points)
    expected: list = []
    full = oracle.forward(made["config"], made["weights"], [1, 2, 3, 250], expected)
    assert row_errors(logits, full).max() < F32_LIMIT and row_errors(taps[(1, "block_output")], expected[1]).max() < F32_LIMIT
    layer = made["config"]["layers"][1]
    mixed = oracle.latent_attention_mixer(expected[0], made["weights"], "l1.mix.", layer["mixer"], 1e-4, sinks=False)
    assert row_errors(taps[(1, "mixer_projection")], mixed).max() < F32_LIMIT
    assert taps[(1, "mixer_output")].shape == (4, 3 * 64)
    c.close()
    for point in ("mixer_filter", "pre_norm"):                       # taps that these blocks have no buffer for
        c = context(rt, made["model"], "float32")
        with pytest.raises(rt.EvoError) as refused:
            c.prefill_with_dumps(b"ab", [(1, point)])
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
