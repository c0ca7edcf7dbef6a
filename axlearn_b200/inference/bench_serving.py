"""Serving throughput of Sagisun and Zukitar beside the Fuji decoder of the same widths (one GPU, random weights).

All models run on their decode engines: prompts of equal length, then greedy decoding from a captured
step.  ``bench.py --serving`` prints one JSON line per (size, model, batch); ``--serving_models`` picks models,
``--serving_table FILE`` adds the device time of every kernel of one prompt pass and one decoding step.  Layers
repeat (Zukitar in threes: two state-space, one latent-attention), so a few of them give the per-layer cost;
the vocabulary product is included once.
"""

from __future__ import annotations

import collections
import functools
import gc
import json
import statistics
from typing import Optional

import torch

from axlearn_b200.common import prng
from axlearn_b200.experiments.text.gpt import sagisun, zukitar
from axlearn_b200.inference.bench_decode import random_weights
from axlearn_b200.inference.decode_engine import DecodeEngine, FujiDims, ModuleDecodeEngine
from axlearn_b200.ops import cuda_ops

# Layers per model and (batch, prompt length, decoding steps) per size.
SIZES = {
    "1B": dict(layers=9, runs=[(1, 2048, 64), (8, 2048, 64), (64, 512, 64)]),
    "7B": dict(layers=6, runs=[(1, 4096, 64), (8, 2048, 64), (64, 512, 64)]),
}


def _module_engine(module, size: str, layers: int, batch: int, max_len: int) -> ModuleDecodeEngine:
    cfg = module.size_config(size)
    cfg["layers"] = cfg["layers"][:layers]
    model = module.model_config(cfg).set(name="model", dtype=torch.bfloat16).instantiate(parent=None)
    params = model.initialize_parameters_recursively(prng.PRNGKey(0), device="cuda")
    return ModuleDecodeEngine(model.decoder, params["decoder"], batch=batch, max_len=max_len, device="cuda")


def _fuji_engine(size: str, layers: int, batch: int, max_len: int) -> DecodeEngine:
    cfg = sagisun.size_config(size)
    left, ff = cfg["layers"][0]["mixer"]["left"], cfg["layers"][0]["mlp"]["ff"]
    dims = FujiDims(num_layers=layers, hidden_dim=cfg["width"], num_heads=left["heads"], num_kv_heads=left["kv_heads"],
                    head_dim=left["dim"], ffn_dim=ff, vocab_size=cfg["vocab"])
    return DecodeEngine(random_weights(dims, rank=0, world=1, device="cuda"), dims, batch=batch, max_len=max_len,
                        device="cuda")


def _time(fn, repeat: int) -> float:
    """Median device time of a call in ms (an allocation that grows the memory pool takes as long as several
    passes and would swamp a mean)."""
    events = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(repeat)]
    torch.cuda.synchronize()
    for start, end in events:
        start.record()
        fn()
        end.record()
    torch.cuda.synchronize()
    return statistics.median(start.elapsed_time(end) for start, end in events)


def _kernel_times(fn) -> list:
    from torch.profiler import ProfilerActivity, profile

    fn()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        fn()
        torch.cuda.synchronize()
    total, count = collections.Counter(), collections.Counter()
    for e in prof.events():
        if e.device_type == torch.autograd.DeviceType.CUDA:
            total[e.name[:110]] += e.device_time
            count[e.name[:110]] += 1
    return [(t, count[n], n) for n, t in total.most_common(24)]


ENGINES = {"zukitar": functools.partial(_module_engine, zukitar), "sagisun": functools.partial(_module_engine, sagisun),
           "fuji": _fuji_engine}


def run(*, steps: int, warmup: int, table: Optional[str] = None, sizes: Optional[list] = None,
        models: Optional[list] = None, emit=print) -> list:
    results = []
    out = open(table, "w", encoding="utf-8") if table else None
    for size in sizes or list(SIZES):
        spec = SIZES[size]
        for name in models or list(ENGINES):
            make = ENGINES[name]
            for batch, prompt, new in spec["runs"]:
                engine = make(size, spec["layers"], batch, prompt + new + 16)
                ids = torch.randint(0, engine.logits.shape[1], (batch, prompt),
                                    generator=torch.Generator().manual_seed(0)).cuda()
                for _ in range(max(3, warmup)):
                    engine.prefill(ids)
                prefill_ms = _time(lambda: engine.prefill(ids), steps)  # pylint: disable=cell-var-from-loop
                engine.decode(8)
                engine.prefill(ids)
                decode_ms = _time(lambda: engine.decode(new), 1) / new  # pylint: disable=cell-var-from-loop
                line = {
                    "metric": "serving throughput", "model": name, "size": size, "layers": spec["layers"],
                    "batch": batch, "prompt_len": prompt, "prefill_ms": round(prefill_ms, 3),
                    "prefill_tokens_per_s": round(batch * prompt / prefill_ms * 1e3), "decode_ms": round(decode_ms, 4),
                    "decode_tokens_per_s": round(batch / decode_ms * 1e3), "dtype": "bf16", "data": "synthetic",
                    "launches_per_step": engine.launches_per_step,
                    "l2": "weights, activations and caches of a pass exceed the 126 MB L2",
                }
                results.append(line)
                emit(json.dumps(line))
                if out is not None:
                    for what, fn in (("prefill", lambda: engine.prefill(ids)), ("decode", lambda: engine.decode(1))):  # pylint: disable=cell-var-from-loop
                        out.write(f"== {size} {name} batch {batch} prompt {prompt}: {what}\n")
                        for t, n, kernel in _kernel_times(fn):
                            out.write(f"{t:10.1f} us {n:4d} x {t / n:9.2f}  {kernel}\n")
                    out.flush()
                del engine
                gc.collect()
                torch.cuda.empty_cache()
    cuda_ops.check_status()
    if out is not None:
        out.close()
    return results
