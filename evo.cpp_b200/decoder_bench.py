"""Throughput of a decoder design beside the framework's closest other model at equal size (bench.py --design).

gigusun: beside a StripedHyena2 stack of the same width, number of blocks and weight count (the decoder's two
feed-forward matrices are half again as wide as the three of the gated MLP).  kikepel: beside a Gigusun stack of
window attention blocks of the same width, heads, head size, window and number of blocks, whose feed-forward has
as many weights as a token meets in Kikepel's.  Random weights and random tokens.  For every width:
prefill at several lengths (token ids on the device, CUDA events on the context's stream), cached decode
(one public decode call per token, greedy, logits to the host), and the time of every operator class with its
algorithmic work against the measured peaks.  Weights and activations exceed the 126 MB L2 in every step.
"""
from __future__ import annotations

import gc
import importlib
import json
import shutil
import tempfile
import time
from pathlib import Path

import numpy as np

ROOT = Path(__file__).resolve().parent.parent
BLOCKS = 12
VOCAB = 512
WINDOW, KEEP = 1024, 4


def shapes(width: int) -> dict:
    """Head layout and feed-forward widths at one model width (head size 128)."""
    heads = width // 128
    inner = {2048: 5632, 4096: 11264}[width]
    return {"width": width, "heads": heads, "inner": inner, "ff": inner * 3 // 2}


def decoder_config(art, width: int, max_positions: int) -> dict:
    s = shapes(width)
    H, mlp = s["heads"], {"kind": "dense", "ff": s["ff"]}
    delta = {"type": "delta", "mlp": mlp,
             "mixer": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4}}
    attention = {"type": "attention", "mlp": mlp,
                 "mixer": {"heads": H, "kv_heads": H // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                           "mask": {"size": WINDOW, "keep_first": KEEP}}}
    gla = {"type": "gla", "mlp": mlp, "mixer": {"heads": H // 2, "dim": 128, "vdim": 256, "tau": 16.0}}
    return art.gigusun_config([(delta, attention, gla)[i % 3] for i in range(BLOCKS)], vocab=VOCAB, width=width,
                              max_positions=max_positions)


LATENT_BLOCKS = 6
LATENT_EXPERTS = {2048: 32, 4096: 16}
LATENT_TOP = 4


def latent_config(art, width: int) -> dict:
    """Kikepel: one dense block, then mixtures of experts; sinks in every other block."""
    s = shapes(width)
    H, experts = s["heads"], LATENT_EXPERTS[width]
    layers = []
    for i in range(LATENT_BLOCKS):
        mlp = {"kind": "dense", "ff": s["inner"]} if i == 0 else {
            "kind": "moe", "expert": {"ff": s["inner"] // LATENT_TOP, "limit": 7.0}, "router": {"experts": experts, "top": LATENT_TOP}}
        layers.append({"type": ("latent_attention", "latent_attention_2")[i % 2], "mlp": mlp,
                       "mixer": {"heads": H, "dim": 128, "vdim": 128, "q_rank": width * 3 // 8, "kv_rank": 512,
                                 "scale": 128 ** -0.5, "mask": {"size": WINDOW}}})
    return art.kikepel_config(layers, vocab=VOCAB, width=width)


def window_stack_config(art, width: int, max_positions: int) -> dict:
    """Gigusun's attention block alone, with a key/value head per query head."""
    s = shapes(width)
    H = s["heads"]
    block = {"type": "attention", "mlp": {"kind": "dense", "ff": s["ff"]},
             "mixer": {"heads": H, "kv_heads": H, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                       "mask": {"size": WINDOW, "keep_first": 0}}}
    return art.gigusun_config([block] * LATENT_BLOCKS, vocab=VOCAB, width=width, max_positions=max_positions)


def seen_keys(tokens: int, context: int, size: int, keep: int = 0) -> int:
    first = context - tokens
    return sum(min(first + i + 1, size) + min(keep, max(0, first + i + 1 - size)) for i in range(tokens))


def latent_work(config: dict, tokens: int, context: int) -> dict:
    """class_work of a Kikepel configuration (prompts: keys and values are expanded from the latents)."""
    D, T = config["width"], tokens
    gemm, grouped, routing, attention = [0.0, 0.0], [0.0, 0.0], [0.0, 0.0], [0.0, 0.0]
    norm_bytes = 6.0 * T * D

    def product(total, rows, k, n, out_bytes):
        total[0] += 2.0 * rows * k * n
        total[1] += 2.0 * k * n + 2.0 * rows * k + rows * n * out_bytes

    product(gemm, T, D, config["vocab"], 4.0)
    for layer in config["layers"]:
        m, mlp = layer["mixer"], layer["mlp"]
        H, dim, vdim, q, c = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
        span = min(context, T + m["mask"]["size"] - 1)
        product(gemm, T, D, q + c, 2.0)
        product(gemm, T, q, H * dim, 2.0)
        product(gemm, span, c, H * dim, 2.0)
        product(gemm, span, c, H * vdim, 2.0)
        product(gemm, T, H * vdim, D, 4.0)
        norm_bytes += 4.0 * T * (q + c) + T * D * (4.0 + 8.0 + 2.0)
        attention[0] += 2.0 * H * (dim + vdim) * seen_keys(T, context, m["mask"]["size"])
        attention[1] += 2.0 * H * (T * (dim + vdim) + span * (dim + vdim))
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            product(gemm, T, D, 2 * mlp["ff"], 1.0)
            product(gemm, T, mlp["ff"], D, 4.0)
            norm_bytes += T * D * (4.0 + 8.0 + 2.0)
            continue
        E, top, ff = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
        pairs = T * top
        grouped[0] += 6.0 * pairs * D * ff
        grouped[1] += 6.0 * min(E, pairs) * D * ff + 2.0 * pairs * (2 * D + 2 * ff)
        product(routing, T, D, E, 4.0)
        routing[1] += 2.0 * T * D + 2.0 * pairs * D
        norm_bytes += T * D * (2.0 * top + 8.0 + 2.0)
    return {"gemm_bf16_tcgen05": (gemm[0], 0.0, gemm[1]), "gemm_grouped": (grouped[0], 0.0, grouped[1]),
            "attention": (attention[0], 0.0, attention[1]), "rms_norm": (0.0, 0.0, norm_bytes),
            "routing": (routing[0], 0.0, routing[1])}


def token_weight_bytes(config: dict, art) -> float:
    """Bytes of the weights that one token meets (its experts' only; one embedding row)."""
    total = 0.0
    for name, shape in art.decoder_manifest(config):
        share = 1.0
        if ".mlp.e" in name:
            router = config["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
            share = router["top"] / router["experts"]
        total += 2.0 * share * (shape[-1] if name in ("embed", "pos") else float(np.prod(shape)))
    return total


def class_work(config: dict, tokens: int, context: int) -> dict:
    """{operator class: (FLOPs on the tensor cores, F32 multiply-adds of the recurrences, HBM bytes)} of one pass
    over `tokens` rows whose last sees `context` keys."""
    D, T = config["width"], tokens
    gemm_flops = 2.0 * T * D * config["vocab"]
    gemm_bytes = 2.0 * D * config["vocab"] + 4.0 * T * config["vocab"]
    norm_bytes = attention_flops = attention_bytes = poly_bytes = 0.0
    linear = [0.0, 0.0]
    delta = [0.0, 0.0]
    for layer in config["layers"]:
        m = layer["mixer"]
        H, dim, vdim = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        if layer["type"] == "attention":
            columns = (H + G) * dim + G * vdim + H
            size, keep = m["mask"]["size"], m["mask"]["keep_first"]
            attention_flops += 2.0 * H * (dim + vdim) * seen_keys(T, context, size, keep)
            keys = min(context, size + keep + T)
            attention_bytes += 2.0 * (T * H * (2 * dim + vdim) + 2 * G * (dim + vdim) * (T + keys))
        elif layer["type"] == "gla":
            columns = 2 * H * dim + 2 * H * vdim + 16
            linear[0] += 3.0 * T * H * dim * vdim
            linear[1] += 2.0 * T * (2 * H * dim + 3 * H * vdim) + 8.0 * H * dim * vdim
        else:
            columns = 2 * G * dim + 2 * H * vdim + 2 * H
            delta[0] += 4.0 * T * H * dim * vdim
            delta[1] += 2.0 * T * (2 * G * dim + 3 * H * vdim) + 8.0 * H * dim * vdim
        out = H * vdim
        for k, n, accumulate in ((D, columns, False), (out, D, True)):
            gemm_flops += 2.0 * T * k * n
            gemm_bytes += 2.0 * k * n + 2.0 * T * k + T * n * (8.0 if accumulate else 2.0)
        norm_bytes += 2 * T * D * 6.0
        ff = layer["mlp"]["ff"]
        for k, n, accumulate in ((D, ff, False), (ff, D, True)):
            gemm_flops += 2.0 * T * k * n
            gemm_bytes += 2.0 * k * n + 2.0 * T * k + T * n * (8.0 if accumulate else 2.0)
        poly_bytes += 4.0 * T * ff
    return {"gemm_bf16_tcgen05": (gemm_flops, 0.0, gemm_bytes), "rms_norm": (0.0, 0.0, norm_bytes),
            "attention": (attention_flops, 0.0, attention_bytes), "gated_linear_attention": (0.0, *linear),
            "gated_delta_rule": (0.0, *delta), "poly_norm": (0.0, 0.0, poly_bytes)}


def roofline_seconds(work: tuple[float, float, float], peaks: dict) -> float:
    flops, fma, nbytes = work
    return max(flops / (peaks["bf16_tflops_sustained"] * 1e12), fma / peaks["fma_per_second"],
               nbytes / (peaks["hbm_gbs"] * 1e9))


def reference_work(width: int, blocks: int, tokens: int) -> dict:
    """The same for the StripedHyena2 stack (blocks cycle HCS, HCM, HCL, attention)."""
    s, T, D = shapes(width), tokens, width
    I = s["inner"]
    flops = blocks * 2.0 * T * (4 * D * D + 3 * D * I) + 2.0 * T * D * VOCAB
    weights = blocks * 2.0 * (4 * D * D + 3 * D * I)
    nbytes = weights + blocks * 2.0 * T * (D + 3 * D + D + 2 * D + D + I + I + 2 * D)
    quarter = blocks / 4
    hyena = 8.0 * T * D * quarter
    return {"gemm_bf16_tcgen05": (flops, 0.0, nbytes), "rms_norm": (0.0, 0.0, blocks * 2 * 4.0 * T * D),
            "attention": (4.0 * D * T * T / 2 * quarter, 0.0, quarter * 2.0 * T * D * 7),
            "hcs_fused_fir": (0.0, 0.0, hyena), "hcm_fused_fir": (0.0, 0.0, hyena),
            "hcl_modal_scan": (0.0, 48.0 * T * D * quarter, hyena)}


def timed_prefill(torch, context, tokens: int, vocab: int, steps: int, warmup: int) -> float:
    ids = torch.randint(0, vocab, (tokens,), dtype=torch.int32, device="cuda")
    stream = torch.cuda.ExternalStream(context.stream())
    torch.cuda.synchronize()
    for _ in range(warmup):
        context.prefill_device(ids.data_ptr(), tokens, True)
    context.synchronize()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record(stream)
    for _ in range(steps):
        context.prefill_device(ids.data_ptr(), tokens, True)
    stop.record(stream)
    context.synchronize()
    return start.elapsed_time(stop) / steps


def operator_times(torch, context, tokens: int, vocab: int, steps: int) -> dict:
    ids = torch.randint(0, vocab, (tokens,), dtype=torch.int32, device="cuda")
    torch.cuda.synchronize()
    context.profile_enable(True)
    for _ in range(steps):
        context.prefill_device(ids.data_ptr(), tokens, True)
    context.synchronize()
    profile = context.profile_read()
    context.profile_enable(False)
    return {name: (ms / steps, count // steps) for name, (ms, count) in profile.items() if count}


def timed_decode(context, prompt: list[int], steps: int) -> float:
    row = context.prefill_tokens(prompt)[-1]
    for _ in range(8):
        row = context.decode(int(row.argmax()))
    begin = time.perf_counter()
    for _ in range(steps):
        row = context.decode(int(row.argmax()))
    return (time.perf_counter() - begin) / steps


def measure(model, flags: int, lengths: list[int], decode_steps: int, steps: int, warmup: int, work, peaks: dict,
            torch, weight_bytes: float | None = None) -> dict:
    context = model.context(max(lengths) + 64, flags)
    vocab = model.vocab
    result = {"prefill": {}, "operators": {}}
    for tokens in lengths:
        ms = timed_prefill(torch, context, tokens, vocab, steps, warmup)
        result["prefill"][str(tokens)] = {"ms": round(ms, 4), "tokens_per_second": round(tokens / ms * 1e3)}
    longest = max(lengths)
    estimates = work(longest)
    for name, (ms, count) in operator_times(torch, context, longest, vocab, steps).items():
        entry = {"ms": round(ms, 4), "launches": count}
        if name in estimates and ms > 0:
            entry["of_roofline"] = round(roofline_seconds(estimates[name], peaks) / (ms * 1e-3), 3)
        result["operators"][name] = entry
    rng = np.random.default_rng(3)
    prompt = [int(t) for t in rng.integers(0, vocab, 1024)]
    if decode_steps:
        seconds = timed_decode(context, prompt, decode_steps)
        read = weight_bytes if weight_bytes is not None else sum(s.weight_bytes for s in context.stages())
        result["decode_after_1024_tokens"] = {"ms_per_token": round(seconds * 1e3, 4),
                                              "tokens_per_second": round(1.0 / seconds, 1), "weight_bytes": read,
                                              "of_weight_stream": round(read / (peaks["hbm_gbs"] * 1e9) / seconds, 3)}
    context.close()
    return result


def decoder_arm(library, art, base: Path, config: dict, work, arguments: tuple, peaks: dict, torch) -> dict:
    lengths, decode_steps, steps, warmup = arguments
    directory = art.write_decoder_random(base / config["architecture"], config, 5, "cuda")
    model = library.load(directory)
    result = measure(model, 0, lengths, decode_steps, steps, warmup, lambda t: work(config, t, t), peaks, torch,
                     token_weight_bytes(config, art))
    model.close()
    shutil.rmtree(directory)
    gc.collect()
    return result


def hyena_arm(library, art, rt, base: Path, width: int, arguments: tuple, peaks: dict, torch) -> dict:
    lengths, decode_steps, steps, warmup = arguments
    s = shapes(width)
    spec = art.fixture_spec(width=width, layers=BLOCKS, heads=s["heads"], inner=s["inner"], hcs_groups=width // 16,
                            hcm_groups=width // 16, vocab=VOCAB)
    path = base / f"hyena-{width}"
    art.write_synthetic(path / "model.safetensors", spec, 6, device="cuda", max_shard_bytes=1 << 40)
    model = library.load(path / "model.safetensors", flags=rt.MODEL_FLAG_ALLOW_SYNTHETIC)
    result = measure(model, rt.CONTEXT_FLAG_TENSORCORE_FP8 | rt.CONTEXT_FLAG_FULL_ARENA, lengths, decode_steps, steps, warmup,
                     lambda t: reference_work(width, BLOCKS, t), peaks, torch)
    model.close()
    shutil.rmtree(path)
    gc.collect()
    return result


def run(package, clock_sampler, steps: int, warmup: int, lengths: list[int], widths: list[int], decode_steps: int,
        design: str = "gigusun") -> dict:
    import torch

    art, rt = (importlib.import_module(f"{package.__name__}.{name}") for name in ("artifact", "runtime"))
    library = rt.EvoLibrary(package.EVO_LIBRARY)
    peaks_file = ROOT / "MEASURED_PEAKS.json"
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops_sustained": 1400.0}
    if peaks_file.exists():
        peaks.update({k: v for k, v in json.loads(peaks_file.read_text()).items() if k in peaks})
    properties = torch.cuda.get_device_properties(0)
    peaks["fma_per_second"] = 128.0 * properties.multi_processor_count * 1.9e9
    line = {"design": design.capitalize(), "dtype": "bf16", "data": "synthetic",
            "blocks": LATENT_BLOCKS if design == "kikepel" else BLOCKS, "steps": steps, "warmup": warmup,
            "window": WINDOW, "keep_first": 0 if design == "kikepel" else KEEP, "peaks": peaks, "sizes": {}}
    base = Path(tempfile.mkdtemp(prefix="decoder_bench_"))
    arguments = (lengths, decode_steps, steps, warmup)
    try:
        with clock_sampler(0) as clocks:
            for width in widths:
                longest = max(lengths)
                result = {"shape": shapes(width)}
                if design == "kikepel":
                    result["shape"].update(experts=LATENT_EXPERTS[width], top=LATENT_TOP)
                    result["kikepel"] = decoder_arm(library, art, base, latent_config(art, width), latent_work, arguments,
                                                    peaks, torch)
                    result["gigusun_attention"] = decoder_arm(library, art, base, window_stack_config(art, width, longest + 64),
                                                              class_work, arguments, peaks, torch)
                else:
                    result["gigusun"] = decoder_arm(library, art, base, decoder_config(art, width, longest + 64), class_work,
                                                    arguments, peaks, torch)
                    result["striped_hyena2"] = hyena_arm(library, art, rt, base, width, arguments, peaks, torch)
                line["sizes"][str(width)] = result
        line["clocks"] = clocks.summary()
    finally:
        shutil.rmtree(base, ignore_errors=True)
    return line
