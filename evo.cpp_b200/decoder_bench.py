"""Throughput of a Gigusun decoder beside a StripedHyena2 stack of equal size (bench.py --design gigusun).

Both models have the same width, number of blocks and weight count (the decoder's two feed-forward matrices
are half again as wide as the three of the gated MLP), random weights and random tokens.  For every width:
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
            first = context - T
            seen = sum(min(first + i + 1, size) + min(keep, max(0, first + i + 1 - size)) for i in range(T))
            attention_flops += 2.0 * H * (dim + vdim) * seen
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
            torch) -> dict:
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
        result["decode_after_1024_tokens"] = {"ms_per_token": round(seconds * 1e3, 4),
                                              "tokens_per_second": round(1.0 / seconds, 1),
                                              "weight_bytes": sum(s.weight_bytes for s in context.stages()),
                                              "of_weight_stream": round(sum(s.weight_bytes for s in context.stages()) /
                                                                        (peaks["hbm_gbs"] * 1e9) / seconds, 3)}
    context.close()
    return result


def run(package, clock_sampler, steps: int, warmup: int, lengths: list[int], widths: list[int], decode_steps: int) -> dict:
    import torch

    art, rt = (importlib.import_module(f"{package.__name__}.{name}") for name in ("artifact", "runtime"))
    library = rt.EvoLibrary(package.EVO_LIBRARY)
    peaks_file = ROOT / "MEASURED_PEAKS.json"
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops_sustained": 1400.0}
    if peaks_file.exists():
        peaks.update({k: v for k, v in json.loads(peaks_file.read_text()).items() if k in peaks})
    properties = torch.cuda.get_device_properties(0)
    peaks["fma_per_second"] = 128.0 * properties.multi_processor_count * 1.9e9
    line = {"design": "Gigusun", "dtype": "bf16", "data": "synthetic", "blocks": BLOCKS, "steps": steps, "warmup": warmup,
            "window": WINDOW, "keep_first": KEEP, "peaks": peaks, "sizes": {}}
    base = Path(tempfile.mkdtemp(prefix="decoder_bench_"))
    try:
        with clock_sampler(0) as clocks:
            for width in widths:
                s = shapes(width)
                longest = max(lengths)
                config = decoder_config(art, width, longest + 64)
                directory = art.write_gigusun_random(base / f"decoder-{width}", config, 5, "cuda")
                model = library.load(directory)
                decoder = measure(model, 0, lengths, decode_steps, steps, warmup,
                                  lambda t: class_work(config, t, t), peaks, torch)
                model.close()
                shutil.rmtree(directory)
                spec = art.fixture_spec(width=width, layers=BLOCKS, heads=s["heads"], inner=s["inner"],
                                        hcs_groups=width // 16, hcm_groups=width // 16, vocab=VOCAB)
                path = base / f"hyena-{width}"
                art.write_synthetic(path / "model.safetensors", spec, 6, device="cuda", max_shard_bytes=1 << 40)
                model = library.load(path / "model.safetensors", flags=rt.MODEL_FLAG_ALLOW_SYNTHETIC)
                hyena = measure(model, rt.CONTEXT_FLAG_TENSORCORE_FP8 | rt.CONTEXT_FLAG_FULL_ARENA, lengths, decode_steps,
                                steps, warmup, lambda t: reference_work(width, BLOCKS, t), peaks, torch)
                model.close()
                shutil.rmtree(path)
                gc.collect()
                line["sizes"][str(width)] = {"shape": s, "gigusun": decoder, "striped_hyena2": hyena}
        line["clocks"] = clocks.summary()
    finally:
        shutil.rmtree(base, ignore_errors=True)
    return line
