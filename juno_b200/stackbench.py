"""Prefill and decode throughput of a registered design (random weights) beside the framework's LLaMA family at equal size.

    python bench.py --design vosotar|desilorn [--sizes small,medium,large] [--steps K] [--warmup W]

Equal size: the same width, feed-forward width, layers, vocabulary and number of query heads; the LLaMA model is Q4_K_M, as the
framework serves it.  Timed with CUDA events on the context's stream after warm-up; the weights of a step exceed L2.
"""
from __future__ import annotations

import os
import shutil
import tempfile

import numpy as np

from . import synth
from .handler import B200TransformerHandler
from .matvec import GpuContext
from .safetensors_file import write_model_folder

# width, heads, feed-forward, q_rank, kv_rank, layers (heads of 128; grouped attention has 8 key/value heads, as LLaMA)
SIZES = {"small": (2048, 16, 8192, 768, 512, 8), "medium": (4096, 32, 14336, 1536, 512, 4), "large": (8192, 64, 28672, 1536, 512, 2)}
VOCAB = 32000


def vosotar_model(size: str) -> dict:
    w, heads, ff, qr, kr, n = SIZES[size]
    one = dict(heads=heads, dim=128, vdim=128, q_rank=qr, kv_rank=kr, scale=128 ** -0.5, ff=ff)
    return synth.vosotar_config(w, VOCAB, [dict(one) for _ in range(n)])


def desilorn_model(size: str) -> dict:
    """Window and chunk layers in turn, spans longer than the measured contexts (every cached key is read, as in LLaMA)."""
    w, heads, ff, _, _, n = SIZES[size]
    one = dict(heads=heads, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, ff=ff)
    kinds = (dict(one, size=8192, rot=(500000.0, 128)), dict(one, size=4096, q_temp=(0.1, 1024)))
    return synth.desilorn_config(w, VOCAB, [dict(kinds[i % 2]) for i in range(n)], streams=4)


DESIGNS = {"vosotar": (vosotar_model, synth.vosotar_shapes, synth.random_vosotar),
           "desilorn": (desilorn_model, synth.desilorn_shapes, synth.random_desilorn)}


def llama_arch(size: str) -> synth.Arch:
    w, heads, ff, _, _, n = SIZES[size]
    return synth.Arch(w, n, heads, 8, ff, VOCAB, 1e-5, 500000.0)


def matrix_params(shapes: dict) -> float:
    """Weights every position of a prompt meets in matrix products, layers only."""
    return float(sum(np.prod(s) for n, (s, fan) in shapes.items() if n.startswith("l") and len(s) == 2 and fan and "canon" not in n))


def _events():
    import torch
    return torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)


def time_prefill(h, ctx, tokens: int, warmup: int, steps: int) -> float:
    """ms of one pass over a prompt of `tokens` positions (the same request again from position 0)."""
    import torch
    stream = torch.cuda.ExternalStream(ctx.stream())
    ids = np.random.default_rng(1).integers(0, VOCAB, tokens).tolist()
    for _ in range(warmup):
        h.prefill("p", ids, 0)
    e0, e1 = _events()
    torch.cuda.synchronize()
    e0.record(stream)
    for _ in range(steps):
        h.prefill("p", ids, 0)
    e1.record(stream)
    torch.cuda.synchronize()
    h.evict("p")
    return e0.elapsed_time(e1) / steps


def time_decode(h, ctx, batch: int, context: int, warmup: int, steps: int):
    """ms of one decode step of `batch` requests at `context` positions, the greedy loop kept on the device."""
    import torch
    stream = torch.cuda.ExternalStream(ctx.stream())
    ids = np.random.default_rng(2).integers(0, VOCAB, context).tolist()
    names = [f"d{i}" for i in range(batch)]
    for n in names:
        h.prefill(n, ids, 0)
    last = h.decode_greedy(names, [1] * batch, [context] * batch, steps)[-1].tolist()  # sizes the id buffer
    last = h.decode_greedy(names, last, [context + steps] * batch, warmup)[-1].tolist()
    e0, e1 = _events()
    torch.cuda.synchronize()
    e0.record(stream)
    h.decode_greedy(names, last, [context + steps + warmup] * batch, steps)
    e1.record(stream)
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    # shares of the step, with events round every launch (graphs off)
    ctx.profile(True)
    ctx.profile_read()
    h.forward_batch(names, [[1]] * batch, [context + 2 * steps + warmup] * batch, want_logits=False, want_argmax=True)
    prof = {k: {"launches": v["launches"], "ms": round(v["ms"], 4)} for k, v in ctx.profile_read().items() if v["launches"]}
    ctx.profile(False)
    for n in names:
        h.evict(n)
    return ms, prof


def measure(h, ctx, batches, context: int, warmup: int, steps: int, prefill_steps: int) -> dict:
    out = {"prefill": {}, "decode": {}}
    ms = time_prefill(h, ctx, context, 2, prefill_steps)
    out["prefill"] = {"tokens": context, "ms": ms, "tokens_per_s": context / ms * 1e3}
    ctx.profile(True)
    ctx.profile_read()
    h.prefill("q", np.random.default_rng(1).integers(0, VOCAB, context).tolist(), 0)
    out["prefill"]["profile"] = {k: {"launches": v["launches"], "ms": round(v["ms"], 4)} for k, v in ctx.profile_read().items() if v["launches"]}
    ctx.profile(False)
    h.evict("q")
    for b in batches:
        ms, prof = time_decode(h, ctx, b, context, warmup, steps)
        out["decode"][str(b)] = {"ms_per_step": ms, "tokens_per_s": b / ms * 1e3, "profile": prof}
    return out


def run(design: str, sizes, batches, context: int, steps: int, warmup: int, peaks: dict, llama: bool = True) -> dict:
    model, shapes, random_model = DESIGNS[design]
    ctx = GpuContext.shared(0)
    res = {}
    hbm, tf = peaks["hbm_gbs"], peaks["bf16_tflops"]
    room = context + 2 * steps + warmup + 16
    for size in sizes:
        cfg = model(size)
        d = tempfile.mkdtemp(prefix="stackbench")
        try:
            write_model_folder(d, cfg, random_model(cfg, 7, fast=True))
            h = B200TransformerHandler.open(d, ctx, max_batch=max(batches), max_seqs=max(batches) + 1, max_ctx=room)
        finally:
            shutil.rmtree(d, ignore_errors=True)
        r = measure(h, ctx, batches, context, warmup, steps, 5)
        m = cfg["layers"][0]["mixer"]
        n_layers, H = len(cfg["layers"]), m["heads"]
        attn = 2.0 * context * context / 2 * H * (m["dim"] + m["vdim"]) * n_layers
        flops = 2.0 * context * matrix_params(shapes(cfg)) + attn
        r["prefill"]["tflops"] = flops / r["prefill"]["ms"] / 1e9
        r["prefill"]["of_measured"] = r["prefill"]["tflops"] / tf
        r["prefill"]["attention_tflops"] = attn / r["prefill"]["profile"]["attention"]["ms"] / 1e9
        for b, v in r["decode"].items():
            nbytes = h.arch.weight_bytes + int(b) * (context + 1.5 * steps + warmup) * h.arch.cache_bytes_per_token
            v["gbs"] = nbytes / v["ms_per_step"] / 1e6
            v["of_measured"] = v["gbs"] / hbm
            v["attention_gbs"] = int(b) * (context + 2 * steps + warmup) * h.arch.cache_bytes_per_token / v["profile"]["attention"]["ms"] / 1e6
        h.release_gpu_resources()
        res[size] = {design: r}
        if not llama:
            continue
        arch = llama_arch(size)
        h = B200TransformerHandler(arch, ctx, max_batch=max(64, max(batches)), max_seqs=max(batches) + 1, max_ctx=room, kv_dtype="f16")
        h.load(synth.random_model(arch, 7))
        r = measure(h, ctx, batches, context, warmup, steps, 2)
        bpw = {synth.Q4_K: 144 / 256, synth.Q6_K: 210 / 256, synth.Q8_0: 34 / 32}
        kinds = (synth.T_ATTN_Q, synth.T_ATTN_K, synth.T_ATTN_V, synth.T_ATTN_OUT, synth.T_FFN_GATE, synth.T_FFN_UP, synth.T_FFN_DOWN)
        params = sum(float(np.prod(synth.tensor_shape(arch, k))) for k in kinds) * arch.n_layers
        wb = sum(float(np.prod(synth.tensor_shape(arch, k))) * bpw[synth.q4_k_m_type(k)] for k in kinds) * arch.n_layers
        wb += float(np.prod(synth.tensor_shape(arch, synth.T_OUTPUT))) * bpw[synth.q4_k_m_type(synth.T_OUTPUT)]
        flops = 2.0 * context * params + 2.0 * context * context * arch.hidden * arch.n_layers
        r["prefill"]["tflops"] = flops / r["prefill"]["ms"] / 1e9
        r["prefill"]["of_measured"] = r["prefill"]["tflops"] / tf
        for b, v in r["decode"].items():
            nbytes = wb + int(b) * (context + 1.5 * steps + warmup) * 4.0 * arch.kv_dim * arch.n_layers
            v["gbs"] = nbytes / v["ms_per_step"] / 1e6
            v["of_measured"] = v["gbs"] / hbm
            v["attention_gbs"] = int(b) * (context + 2 * steps + warmup) * 4.0 * arch.kv_dim * arch.n_layers / v["profile"]["attention"]["ms"] / 1e6
        h.release_gpu_resources()
        res[size]["llama_q4_k_m"] = r
    return res
