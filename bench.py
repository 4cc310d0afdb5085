"""Measures decode and prefill throughput of the engine on one B200 and prints ONE JSON line.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

The model has the layer sizes of TinyLlama 1.1B (22 layers, hidden 2048, 32 heads, 4 key/value
heads, head size 64, feed-forward 5632, vocabulary 32000) with random weights N(0, 0.02) and
seeded random token ids.  A "step" is one decode step of a batch of 8 requests whose prompts of
512 tokens were prefilled before the clock starts.  ``value`` is decoded tokens a second over
exactly K steps, timed on the device with CUDA events; ``e2e`` is the same through the Python
entry point ``LLM.generate`` (host token ids in, host token ids out, every step's descriptor
copied from pinned memory and its tokens read back).  ``prefill`` is one prompt of 2,048
tokens; ``roofline`` relates the bytes a decode step has to read (every weight once, and the
cache of the live requests) to its time; ``points`` holds decode at batch 1 and 64.
Peaks come from MEASURED_PEAKS.json beside this file when present, else from an earlier
measurement on the same pool (and the line says which).

``python bench.py --design nurolorn-small|nurolorn-1b|kafepel-small|kafepel-1b|nudodra-small|nudodra-1b|tenotar-small|tenotar-1b|pefedra-small|pefedra-1b|zifuzen-small|zifuzen-1b`` prints, instead of the line, prefill and decode
throughput of that configuration beside a Llama of equal width, depth and feed-forward size, and the design's kernels against
their rooflines.

``python bench.py --sweep [--steps K]`` prints no JSON line but two tables: decode steps over batch sizes and
context lengths, and prefills over prompt lengths, timed the same way.
"""

from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}
MODEL = "tinyllama-1.1b"
PROMPT_LEN, NEW_TOKENS, PREFILL_TOKENS = 512, 256, 2048


def load_peaks() -> tuple[dict, str]:
    path = ROOT / "MEASURED_PEAKS.json"
    if path.is_file():
        try:
            d = json.loads(path.read_text())
            flat = {}

            def walk(x):
                if isinstance(x, dict):
                    for k, v in x.items():
                        if isinstance(v, (int, float)) and k in FALLBACK_PEAKS:
                            flat[k] = float(v)
                        else:
                            walk(v)

            walk(d)
            if "hbm_gbs" in flat and "bf16_tflops" in flat:
                return {**FALLBACK_PEAKS, **flat}, "measured"
        except (ValueError, OSError):
            pass
    return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index = index
        self.proc = None
        self.lines: list[tuple[float, str]] = []
        self.window = [0.0, float("inf")]  # only samples taken while the timed region ran are counted

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "20"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append((time.time(), line.strip()))

    def begin(self):
        self.window[0] = time.time()

    def end(self):
        self.window[1] = time.time()

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self) -> dict:
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for stamp, line in self.lines:
            if not self.window[0] <= stamp <= self.window[1] + 0.02:
                continue
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 6:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for name, flag in zip(names, parts[2:6]):
                if flag.lower().startswith("active"):
                    reasons.add(name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


def reference_arm(args) -> int:
    """The unmodified reference from ``baseline/_ref`` through its own public API."""
    ref = ROOT / "baseline" / "_ref"
    if not (ref / "llmserve").is_dir():
        print(json.dumps({"impl": "reference", "unavailable": "the reference is not installed under baseline/_ref (pip install --no-index --target baseline/_ref failed or was not run)"}))
        return 0
    sys.path.insert(0, str(ref))
    try:
        import torch
        from llmserve.config import ModelConfig
        from llmserve.datatypes import SamplingParams as RefParams
        from llmserve.kvcache.paged import PagedKVCache
        from llmserve.scheduler.engine import ContinuousBatchingEngine
        from llmserve.weights import random_model as ref_random_model
    except Exception as e:  # noqa: BLE001
        print(json.dumps({"impl": "reference", "unavailable": f"the reference does not import here: {type(e).__name__}: {e}"[:300]}))
        return 0
    if not torch.cuda.is_available():
        print(json.dumps({"impl": "reference", "unavailable": "no CUDA device"}))
        return 0
    batch, steps, warmup = 8, args.steps, args.warmup
    cfg = ModelConfig()  # the reference's defaults are TinyLlama 1.1B's sizes
    model = ref_random_model(cfg, seed=0, device="cuda", dtype=torch.bfloat16, std=0.02)
    total_new = warmup + steps + 1
    cache = PagedKVCache(cfg, num_blocks=batch * (-(-(PROMPT_LEN + total_new) // 16) + 1) + 8, block_size=16, device="cuda", dtype=torch.bfloat16)
    engine = ContinuousBatchingEngine(model, cache, max_batch_size=batch, max_prefill_tokens=batch * PROMPT_LEN)
    g = torch.Generator().manual_seed(1)
    for _ in range(batch):
        engine.add_request(torch.randint(0, cfg.vocab_size, (PROMPT_LEN,), generator=g).tolist(), RefParams(max_new_tokens=total_new))
    engine.step()  # prefill of all eight, first token
    for _ in range(warmup):
        engine.step()
    torch.cuda.synchronize()
    with ClockSampler() as clocks:
        t0 = time.perf_counter()
        for _ in range(steps):
            engine.step()  # one decode pass; ends in a host read of the tokens
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
    value = batch * steps / dt
    print(json.dumps({
        "impl": "reference", "metric": "decode_tokens_per_s", "value": value, "unit": "tokens/s", "n_gpus": 1, "steps": steps,
        "warmup": warmup, "ms_per_step": dt / steps * 1e3, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic", "clocks": clocks.summary(),
        "e2e": {"value": value, "unit": "tokens/s", "h2d_bytes_per_step": None, "d2h_bytes_per_step": batch * 8},
        "config": {"model": "TinyLlama-1.1B sizes, random weights", "global_batch": batch, "seq_len": 2048, "prompt_len": PROMPT_LEN,
                   "parallelism": "single GPU", "api": "ContinuousBatchingEngine.step", "timing": "wall clock around K engine steps"},
    }))
    return 0


def model_numbers(cfg) -> dict:
    h, L, H, KV, D = cfg.hidden_size, cfg.num_hidden_layers, cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim
    I, V = cfg.intermediate_size, cfg.vocab_size
    layer_params = h * (H + 2 * KV) * D + H * D * h + 3 * h * I
    return {"layer_params": layer_params, "head_params": V * h, "kv_bytes_per_token": 2 * L * KV * D * 2, "L": L, "H": H, "D": D}


def prefill_flops(cfg, tokens: int) -> float:
    m = model_numbers(cfg)
    gemm = 2.0 * tokens * m["layer_params"] * m["L"] + 2.0 * m["head_params"]
    attention = m["L"] * 4.0 * m["H"] * m["D"] * tokens * (tokens + 1) / 2.0
    return gemm + attention


def design_comparison(args) -> int:
    """Prefill and decode of a preset of another design beside a Llama twin (the same width, as many layers as the design runs
    entries of its order, a SwiGLU feed-forward of the same parameter count, vocabulary and head size alike), both with
    random weights, through the same step function; then the design's kernels one by one against their rooflines.
    Every timed launch follows a write of 256 MB (larger than L2); times are CUDA events on the launching stream."""
    import torch

    from llmserve_triton_kernels_b200 import models as _models  # noqa: F401
    from llmserve_triton_kernels_b200 import ops
    from llmserve_triton_kernels_b200.cache import CacheManager
    from llmserve_triton_kernels_b200.config import architecture_of
    from llmserve_triton_kernels_b200.config.presets import PRESETS
    from llmserve_triton_kernels_b200.engine.batch import StepEntry
    from llmserve_triton_kernels_b200.engine.step import StepFunction
    from llmserve_triton_kernels_b200.models.load import random_model

    peaks, peaks_from = load_peaks()
    device = "cuda:0"
    torch.cuda.set_device(device)
    design = dict(PRESETS[args.design])
    arch = architecture_of(design)
    dcfg = arch.config_class.from_dict(design)
    entries = len(arch.plan(dcfg).schedule)
    width, vocab = design["width"], design["vocab"]
    nudodra = design["architecture"] == "Nudodra"
    tenotar = design["architecture"] == "Tenotar"
    pefedra = design["architecture"] == "Pefedra"
    zifuzen = design["architecture"] == "Zifuzen"
    if nudodra or tenotar or zifuzen:  # no dense feed-forward (or one layer's only): the twin's has the size of what a token uses (its chosen experts and the shared one)
        moe = next(x["mlp"] for x in design["layers"] if x.get("mlp") and x["mlp"].get("kind", "moe") == "moe")
        ff = moe["router"]["top"] * moe["expert"]["ff"] + (moe["shared"]["ff"] if moe.get("shared") else 0)
    else:
        ff = next(x["mlp"]["ff"] for x in design["layers"] if x.get("mlp") and "ff" in x["mlp"])
    gated = design["architecture"] in ("Kafepel", "Nudodra", "Tenotar", "Zifuzen")  # their feed-forwards have three matrices, like the twin's
    twin = {
        "architectures": ["LlamaForCausalLM"], "model_type": "llama", "hidden_act": "silu", "rope_theta": 10000.0, "rms_norm_eps": 1e-5,
        "tie_word_embeddings": False, "vocab_size": vocab, "hidden_size": width, "intermediate_size": ff if gated else (ff * 2 // 3 + 63) // 64 * 64,
        "num_hidden_layers": entries, "num_attention_heads": width // 64, "num_key_value_heads": max(1, width // 512),
        "max_position_embeddings": 8192,
    }
    flush = torch.empty(256 * 2**20, dtype=torch.uint8, device=device)
    steps = max(3, min(args.steps, 50))

    def timed(fn, n=steps, setup=None):
        total = 0.0
        for i in range(args.warmup + n):
            if setup is not None:
                setup()
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            b.synchronize()
            if i >= args.warmup:
                total += a.elapsed_time(b)
        return total / n * 1e3  # microseconds

    def tokens(n, seed):
        g = torch.Generator().manual_seed(seed)
        return torch.randint(0, vocab, (n,), generator=g).tolist()

    out = {"design": args.design, "peaks_from": peaks_from, "models": {}}
    compared = [(args.design, design), ("llama-twin", twin)]
    if nudodra:  # the closest design the engine has: side-by-side mixers and a routed feed-forward at the same sizes
        compared.insert(1, (args.design.replace("nudodra", "kafepel"), dict(PRESETS[args.design.replace("nudodra", "kafepel")])))
    if tenotar:  # the closest design the engine has: the same softmax attention part and a mixture of gated experts at the same sizes
        compared.insert(1, (args.design.replace("tenotar", "nudodra"), dict(PRESETS[args.design.replace("tenotar", "nudodra")])))
    if pefedra:  # the closest design the engine has, the same softmax attention part over a window, with a dense feed-forward of as many weights
        span = design["layers"][0]["mixer"]["mask"]["size"]
        m = next(x["mixer"] for x in design["layers"] if x["type"] == "attention_2")
        mixer = {"heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"],
                 "mask": {"size": span, "keep_first": 16}, "rot": {"base": 10000.0, "dims": m["dim"]}}
        compared.insert(1, ("tenotar-twin", {
            "architecture": "Tenotar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [{"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": twin["intermediate_size"]}} for _ in design["layers"]]}))
    if zifuzen:  # the closest design the engine has: a gated recurrence and softmax attention with shared pages, bounded gated experts, at the same sizes
        compared.insert(1, (args.design.replace("zifuzen", "nudodra"), dict(PRESETS[args.design.replace("zifuzen", "nudodra")])))
    for name, cfg_dict in compared:
        a = architecture_of(cfg_dict)
        model = random_model(a.config_class.from_dict(cfg_dict), 0, "bfloat16", device)
        cache = CacheManager(model.cache_specs(), model.plan.schedule, page_size=16, num_pages=8 * 200 + 64, max_requests=8,
                             dtype=torch.bfloat16, device=device)
        step = StepFunction(model, cache)
        res = {"weight_GB": round(model.weight_bytes() / 1e9, 3), "entries_of_the_order": len(model.plan.schedule)}
        for n in (512, 2048):
            toks = tokens(n, n)

            def prefill():
                step([StepEntry("p", toks, [n - 1])])

            def done():
                if cache.has_request("p"):
                    cache.free_request("p")

            us = timed(prefill, setup=done)
            done()
            res[f"prefill_{n}"] = {"ms": round(us / 1e3, 3), "tok_s": round(n / us * 1e6)}
        for batch in (1, 8):
            reqs = [f"d{i}" for i in range(batch)]
            step([StepEntry(r, tokens(512, 7 + i), [511]) for i, r in enumerate(reqs)])
            nxt = tokens(batch, 99)
            us = timed(lambda: step([StepEntry(r, [t], [0]) for r, t in zip(reqs, nxt)]), n=min(100, 8 * steps))
            for r in reqs:
                cache.free_request(r)
            bytes_read = model.weight_bytes() + cache.nbytes() * 0  # weights dominate at 512 tokens of context
            res[f"decode_batch{batch}_ctx512"] = {"ms_per_step": round(us / 1e3, 4), "tok_s": round(batch / us * 1e6),
                                                  "of_hbm_peak_weights_only": round(bytes_read / (us * 1e-6) / 1e9 / peaks["hbm_gbs"], 3)}
        out["models"][name] = res
        del step, cache, model
        torch.cuda.empty_cache()

    # the design's own kernels, alone, at the preset's sizes: 2,048 prompt tokens of one request, and 8 decoding requests
    # of 2,048 cached tokens; a Llama layer's like kernel beside each
    from types import SimpleNamespace

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=device)

    def ctx_for(query_lens, context_lens, page_size=16):
        cu = [0]
        for q in query_lens:
            cu.append(cu[-1] + q)
        width_ = max(-(-c // page_size) for c in context_lens)
        table, page = torch.zeros((len(query_lens), width_), dtype=torch.int32), 0
        owner, pos, slots = [], [], []
        for r, (q, c) in enumerate(zip(query_lens, context_lens)):
            pages = list(range(page, page + -(-c // page_size)))
            page += len(pages)
            table[r, : len(pages)] = torch.tensor(pages, dtype=torch.int32)
            owner += [r] * q
            pos += list(range(c - q, c))
            slots += [pages[p // page_size] * page_size + p % page_size for p in range(c - q, c)]
        ctx = SimpleNamespace(num_tokens=cu[-1], num_requests=len(query_lens), token_request=i32(owner), cu_tokens=i32(cu),
                              context_lens=i32(context_lens), positions=i32(pos), max_query_len=max(query_lens),
                              max_context_len=max(context_lens), host_cu_tokens=cu)
        return ctx, table.to(device), i32(slots), page

    def hbm(name, us, nbytes, like=None):
        kernels[name] = {"us": round(us, 2), "GB_s": round(nbytes / us / 1e3), "of_hbm_peak": round(nbytes / us / 1e3 / peaks["hbm_gbs"], 3)}
        if like:
            kernels[name]["like"] = like

    def tensor(name, us, flops, like=None):
        kernels[name] = {"us": round(us, 2), "TFLOP_s": round(flops / us / 1e6, 1), "of_bf16_peak": round(flops / us / 1e6 / peaks["bf16_tflops"], 3)}
        if like:
            kernels[name]["like"] = like

    bf = torch.bfloat16
    kernels = {}
    if design["architecture"] in ("Kafepel", "Nudodra", "Tenotar", "Pefedra", "Zifuzen"):
        (_zifuzen_kernels if zifuzen else _pefedra_kernels if pefedra else _tenotar_kernels if tenotar else _nudodra_kernels if nudodra else _kafepel_kernels)(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device)
        out["kernels"] = kernels
        out["peaks"] = {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"]}
        print(json.dumps(out, indent=1))
        return 0
    L = next(x["mixer"] for x in design["layers"] if x["type"] == "latent_attention")
    W = next(x["mixer"] for x in design["layers"] if x["type"] == "attention")
    H, rank, rot, hd = L["heads"], L["kv_rank"], L["rot_dim"], L["dim"]
    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n = ctx.num_tokens
        pairs = sum(q * c - q * (q - 1) // 2 for q, c in zip(qs, cs))
        plane = torch.randn(pages, 16, rank + rot, device=device).to(bf)
        q_lat, q_rot = torch.randn(n, H, rank, device=device).to(bf) * 0.1, torch.randn(n, H, rot, device=device).to(bf) * 0.1
        us = timed(lambda: ops.latent_paged_attention(q_lat, q_rot, plane, table, ctx, rank=rank, scale=0.1))
        if label.startswith("prefill"):
            tensor(f"latent_attention_{label}", us, 2.0 * H * (2 * rank + rot) * pairs, like="Llama prefill attention (tcgen05)")
        else:
            hbm(f"latent_attention_{label}", us, sum(cs) * (rank + rot) * 2, like="Llama decode attention (split keys)")
        KV, win = W["kv_heads"], W["mask"]["size"]
        pool = torch.randn(pages, 2, KV, 16, hd, device=device).to(bf)
        qkv = torch.randn(n, (W["heads"] + 2 * KV) * hd, device=device).to(bf)
        slopes = torch.pow(2.0, -8.0 * torch.arange(1, W["heads"] + 1) / W["heads"]).float().to(device)
        kw = dict(num_heads=W["heads"], num_kv_heads=KV, key_dim=hd, value_dim=hd, scale=0.1, window=win, slopes=slopes)
        us = timed(lambda: ops.biased_paged_attention(qkv, pool, table, ctx, **kw))
        seen = sum(min(win, p + 1) for q, c in zip(qs, cs) for p in range(c - q, c))
        if label.startswith("prefill"):
            tensor(f"window_attention_{label}", us, 4.0 * W["heads"] * hd * seen, like="Llama prefill attention (tcgen05)")
        else:
            hbm(f"window_attention_{label}", us, len(qs) * min(win, cs[0]) * 2 * KV * hd * 2, like="Llama decode attention (split keys)")
        # the Llama twin's attention on the same tokens
        tH, tKV = twin["num_attention_heads"], twin["num_key_value_heads"]
        tpool = torch.randn(pages, 2, tKV, 16, 64, device=device).to(bf)
        tq = torch.randn(n, (tH + 2 * tKV) * 64, device=device).to(bf)
        us = timed(lambda: ops.paged_attention(tq, tpool, table, ctx, num_heads=tH, num_kv_heads=tKV, head_dim=64, scale=0.125))
        if label.startswith("prefill"):
            tensor(f"llama_attention_{label}", us, 4.0 * tH * 64 * pairs)
        else:
            hbm(f"llama_attention_{label}", us, sum(cs) * 2 * tKV * 64 * 2)
        # row-wise kernels
        gw = next(x["mixer"]["width"] for x in design["layers"] if x["type"] == "mingru")
        proj = torch.randn(n, 3 * gw, device=device)
        states, sl = torch.zeros(8, gw, device=device), i32(list(range(len(qs))))
        us = timed(lambda: ops.mingru_scan(proj, None, None, states, sl, ctx.cu_tokens, len(qs), gw, bf, max(qs)))
        hbm(f"mingru_scan_{label}", us, n * gw * (12 + 2), like="(no like kernel in Llama)")
        resid, delta, wn = torch.randn(n, width, device=device), torch.randn(n, width, device=device), torch.ones(width, device=device)
        us = timed(lambda: ops.group_rmsnorm(resid, wn, 1e-6, 2, delta=delta, alpha=0.7, out_dtype=bf))
        hbm(f"group_rmsnorm_{label}", us, n * width * (4 + 4 + 4 + 2), like="llama_rmsnorm")
        us = timed(lambda: ops.rmsnorm(resid, wn, 1e-6, delta=delta, out_dtype=bf))
        hbm(f"llama_rmsnorm_{label}", us, n * width * (4 + 4 + 4 + 2))
        stacked = torch.randn(n, H * (hd + rot) + rank + rot + H * hd, device=device).to(bf)
        freq = torch.ones(rot // 2, device=device)
        us = timed(lambda: ops.latent_prepare(stacked, ctx.positions, slots, plane, wn[:rank].contiguous(), freq, 1e-6, H, hd, rot, rank))
        hbm(f"latent_prepare_{label}", us, n * (H * rot * 4 + (rank + rot) * 4), like="llama_rope_kv_write")
        table_r = torch.randn(4096, 64, device=device)
        us = timed(lambda: ops.rope_kv_write(tq, ctx.positions, table_r, slots, tpool, tH, tKV, 64))
        hbm(f"llama_rope_kv_write_{label}", us, n * ((tH + tKV) * 64 * 4 + tKV * 64 * 4))
        up = torch.randn(n, ff, device=device).to(bf)
        us = timed(lambda: ops.unary(up, "relu2"))
        hbm(f"relu2_{label}", us, n * ff * 4, like="llama_swiglu")
        gu = torch.randn(n, 2 * twin["intermediate_size"], device=device).to(bf)
        us = timed(lambda: ops.swiglu(gu))
        hbm(f"llama_swiglu_{label}", us, n * twin["intermediate_size"] * 6)
    out["kernels"] = kernels
    out["peaks"] = {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"]}
    print(json.dumps(out, indent=1))
    return 0


def _kafepel_kernels(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device) -> None:
    """The Kafepel design's own kernels, alone, at the preset's sizes: one request of 2,048 prompt tokens, and 8 decoding
    requests of 2,048 cached tokens; the Llama twin's like kernel beside each."""
    bf = torch.bfloat16
    first = design["layers"][0]["mixer"]
    A, R = first["left"], first["right"]
    moe = next(x["mlp"] for x in design["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe")
    width = design["width"]
    H, KV, D, V = A["heads"], A["kv_heads"], A["dim"], A["vdim"]
    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n = ctx.num_tokens
        pairs = sum(q * c - q * (q - 1) // 2 for q, c in zip(qs, cs))
        prefill = label.startswith("prefill")
        pool = torch.randn(pages, 2, KV, 16, max(D, V), device=device).to(bf)
        q = (torch.randn(n, H * D, device=device) * 0.3).to(bf)
        bias, mix = torch.zeros(H, device=device), torch.randn(H, H, device=device)
        kw = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=A["scale"], softcap=A.get("softcap"), head_bias=bias, head_mix=mix)
        us = timed(lambda: ops.sigmoid_attention(q, pool, table, ctx, **kw))
        if prefill:  # the products with keys and values; the mixing of the heads' weights (2 H flops a weight, 32-bit) is not counted
            tensor(f"sigmoid_attention_{label}", us, 2.0 * H * (D + V) * pairs, like="Llama prefill attention (tcgen05)")
        else:
            hbm(f"sigmoid_attention_{label}", us, sum(cs) * KV * (D + V) * 2, like="Llama decode attention (split keys)")
        tH, tKV = twin["num_attention_heads"], twin["num_key_value_heads"]
        tpool = torch.randn(pages, 2, tKV, 16, 64, device=device).to(bf)
        tq = torch.randn(n, (tH + 2 * tKV) * 64, device=device).to(bf)
        us = timed(lambda: ops.paged_attention(tq, tpool, table, ctx, num_heads=tH, num_kv_heads=tKV, head_dim=64, scale=0.125))
        if prefill:
            tensor(f"llama_attention_{label}", us, 4.0 * tH * 64 * pairs)
        else:
            hbm(f"llama_attention_{label}", us, sum(cs) * 2 * tKV * 64 * 2)
        # projections -> queries, keys in their pages
        proj = torch.randn(n, (H + KV) * D + KV * V, device=device)
        freq = torch.rand(D // 2, device=device)
        qw, kwt = torch.ones(H * D, device=device), torch.ones(KV * D, device=device)
        us = timed(lambda: ops.qk_prepare(proj, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, freq=freq, q_weight=qw, k_weight=kwt,
                                          eps=1e-6, pool=pool, slot_map=slots))
        hbm(f"qk_prepare_{label}", us, n * ((H + KV) * D + KV * V) * (4 + 2), like="llama_rope_kv_write")
        table_r = torch.randn(4096, 64, device=device)
        us = timed(lambda: ops.rope_kv_write(tq, ctx.positions, table_r, slots, tpool, tH, tKV, 64))
        hbm(f"llama_rope_kv_write_{label}", us, n * ((tH + tKV) * 64 * 4 + tKV * 64 * 4))
        # retention: the scan and the step behind it
        RH, RD, RV = R["heads"], R["dim"], R["vdim"]
        rq, rk = torch.randn(n, RH * RD, device=device), torch.randn(n, RH * RD, device=device) * RD ** -0.5
        rv = torch.randn(n, RH * RV, device=device)
        decay = torch.tensor(R["decay"], dtype=torch.float32, device=device)
        states, sl = torch.zeros(8, RH, RD, RV, device=device), i32(list(range(len(qs))))
        us = timed(lambda: ops.retention_scan(rq, rk, rv, decay, states, sl, ctx.cu_tokens, len(qs), RH, RD, RV, max(qs)))
        hbm(f"retention_scan_{label}", us, n * RH * (2 * RD + 2 * RV) * 4 + 2 * len(qs) * RH * RD * RV * 4, like="(no like kernel in Llama)")
        o, gate = torch.randn(n, RH, RV, device=device), torch.randn(n, RH * RV, device=device)
        us = timed(lambda: ops.head_norm_gate(o, gate, 1e-6, "silu", bf))
        hbm(f"head_norm_gate_{label}", us, n * RH * RV * (4 + 4 + 2), like="llama_swiglu")
        a, b, wn = torch.randn(n, width, device=device), torch.randn(n, width, device=device), torch.ones(width, device=device)
        us = timed(lambda: ops.branch_norm_sum([a, b], [wn, wn], 1e-6, 0.5))
        hbm(f"branch_norm_sum_{label}", us, n * width * 12, like="llama_rmsnorm")
        resid = torch.randn(n, width, device=device)
        us = timed(lambda: ops.rmsnorm(resid, wn, 1e-6, delta=a, out_dtype=bf))
        hbm(f"llama_rmsnorm_{label}", us, n * width * (4 + 4 + 4 + 2))
        # routed feed-forward: the choice, and the activation with the tokens' weights
        E, top, eff, sff = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
        hx, wr = torch.randn(n, width, device=device).to(bf), torch.randn(E + 1, width, device=device)
        corr = torch.zeros(E, device=device)
        us = timed(lambda: ops.route(hx, wr, corr, E, top, 2.5, False, True))
        hbm(f"router_{label}", us, n * width * 2 + (E + 1) * width * 4 + n * (E + 1) * 4, like="(no like kernel in Llama)")
        weights = ops.route(hx, wr, corr, E, top, 2.5, False, True)
        up = torch.randn(n, E * eff + sff, device=device).to(bf)
        us = timed(lambda: ops.expert_act_scale(up, weights, E, eff, "relu2"))
        hbm(f"expert_act_scale_{label}", us, n * (E * eff + sff) * 4, like="llama_swiglu")
        gu = torch.randn(n, 2 * twin["intermediate_size"], device=device).to(bf)
        us = timed(lambda: ops.swiglu(gu))
        hbm(f"llama_swiglu_{label}", us, n * twin["intermediate_size"] * 6)


def _nudodra_kernels(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device) -> None:
    """The Nudodra design's own kernels, alone, at the preset's sizes: one request of 2,048 prompt tokens, and 8 decoding
    requests of 2,048 cached tokens; beside each the like kernel of the Kafepel design (the closest one the engine has) at
    the same sizes."""
    bf = torch.bfloat16
    par = next(x["mixer"] for x in design["layers"] if x["type"] == "parallel")
    A, R = par["left"], par["right"]
    moe = next(x["mlp"] for x in design["layers"] if x["mlp"])
    width, S = design["width"], design.get("streams") or 1
    H, KV, D, V = A["heads"], A["kv_heads"], A["dim"], A["vdim"]
    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n = ctx.num_tokens
        pairs = sum(q * c - q * (q - 1) // 2 for q, c in zip(qs, cs))
        prefill = label.startswith("prefill")
        pool = torch.randn(pages, 2, KV, 16, max(D, V), device=device).to(bf)
        q = (torch.randn(n, H * D, device=device) * 0.3).to(bf)
        sinks, gate = torch.zeros(H, device=device), torch.randn(n, H * V, device=device)
        kw = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=A["scale"])
        cache_bytes = sum(cs) * KV * (D + V) * 2 + n * H * (D + V) * 2
        for name, more in (("sink_attention", dict(sinks=sinks)), ("gated_attention", dict(gate=gate))):
            us = timed(lambda: ops.paged_softmax_attention(q, pool, table, ctx, **kw, **more))
            (tensor if prefill else hbm)(f"{name}_{label}", us, 2.0 * pairs * H * (D + V) if prefill else cache_bytes, like="sigmoid_attention")
        bias, mix = torch.zeros(H, device=device), torch.randn(H, H, device=device)
        us = timed(lambda: ops.sigmoid_attention(q, pool, table, ctx, **kw, softcap=30.0, head_bias=bias, head_mix=mix))
        (tensor if prefill else hbm)(f"kafepel_sigmoid_attention_{label}", us, 2.0 * pairs * H * (D + V) if prefill else cache_bytes)
        # the heads' preparation (bias, per-head norms, rotation, cache write) beside Kafepel's (norms over whole projections)
        proj = torch.randn(n, (H + KV) * D + KV * V, device=device)
        freq = torch.rand(A["rot"]["dims"] // 2, device=device)
        b_in, qw, kw_ = torch.randn((H + KV) * D, device=device), torch.ones(D, device=device), torch.ones(D, device=device)
        us = timed(lambda: ops.head_prepare(proj, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, bias=b_in, q_weight=qw, k_weight=kw_,
                                            eps=1e-6, freq=freq, values_are_keys=True, pool=pool, slot_map=slots))
        hbm(f"head_prepare_{label}", us, n * ((H + KV) * D * 4 + (H + 2 * KV) * D * 2), like="qk_prepare")
        qwk, kwk = torch.ones(H * D, device=device), torch.ones(KV * D, device=device)
        us = timed(lambda: ops.qk_prepare(proj, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, freq=freq, q_weight=qwk, k_weight=kwk,
                                          eps=1e-6, pool=pool, slot_map=slots))
        hbm(f"kafepel_qk_prepare_{label}", us, n * ((H + KV) * D + KV * V) * (4 + 2))
        # the recurrence: decays per channel and token beside Kafepel's fixed decay per head
        RH, RD, RV = R["heads"], R["dim"], R["vdim"]
        rq, rk, rz = (torch.randn(n, RH * RD, device=device) for _ in range(3))
        rv = torch.randn(n, RH * RV, device=device)
        zb = torch.full((RH * RD,), 3.0, device=device)
        states, sl = torch.zeros(8, RH, RD, RV, device=device), i32(list(range(len(qs))))
        us = timed(lambda: ops.gated_scan(rq, rk, rv, rz, zb, 1.0 / R["tau"], RD ** -0.5, states, sl, ctx.cu_tokens, len(qs), RH, RD, RV, max(qs)))
        scan_bytes = n * RH * (3 * RD + 2 * RV) * 4 + 2 * len(qs) * RH * RD * RV * 4
        hbm(f"gated_scan_{label}", us, scan_bytes, like="retention_scan")
        decay = torch.full((RH,), 0.97, device=device)
        us = timed(lambda: ops.retention_scan(rq, rk, rv, decay, states, sl, ctx.cu_tokens, len(qs), RH, RD, RV, max(qs)))
        hbm(f"kafepel_retention_scan_{label}", us, n * RH * (2 * RD + 2 * RV) * 4 + 2 * len(qs) * RH * RD * RV * 4)
        o, g2, wn = torch.randn(n, RH, RV, device=device), torch.randn(n, RH * RV, device=device), torch.ones(RV, device=device)
        us = timed(lambda: ops.head_norm_gate(o, g2, 1e-6, "silu", bf, weight=wn))
        hbm(f"head_norm_gate_{label}", us, n * RH * RV * (4 + 4 + 2), like="head_norm_gate (the same kernel)")
        # the stream's copies: update, read-in and norm in one pass, beside Kafepel's meeting of branches with sum and norm
        X = torch.randn(S, n, width, device=device)
        a, b, wd = torch.randn(n, width, device=device), torch.randn(n, width, device=device), torch.ones(width, device=device)
        upd = ops.StreamUpdate(ops.WeightedSum([a, b], [0.6, 0.5]), torch.eye(S, device=device).contiguous(), torch.ones(S, device=device))
        rin = torch.ones(S, device=device)
        us = timed(lambda: ops.hyper_mix_norm(X, upd, rin, wd, 1e-6, out_dtype=bf))
        hbm(f"hyper_mix_norm_{label}", us, n * width * (2 * S * 4 + 2 * 4 + 2), like="branch_sum_norm")
        resid = torch.randn(n, width, device=device)
        pend = ops.BranchSum([a, b], [wd, wd], 1e-6, 0.5)
        us = timed(lambda: ops.branch_sum_rmsnorm(pend, resid, wd, 1e-6, bf))
        hbm(f"kafepel_branch_sum_norm_{label}", us, n * width * (4 * 4 + 2))
        # the experts' activation with the table's weights beside Kafepel's with the router's
        E, top, eff, sff = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
        up2 = torch.randn(n, 2 * (E * eff + sff), device=device).to(bf)
        tab = torch.rand(design["vocab"], E, device=device).argsort(dim=1)[:, :top].to(torch.int32).contiguous()
        ids = torch.randint(0, design["vocab"], (n,), device=device, dtype=torch.int32)
        us = timed(lambda: ops.expert_gated_act(up2, E, eff, sff, 7.0, 7.0, 1.702, ids=ids, table=tab))
        hbm(f"expert_gated_act_{label}", us, n * ((top * eff + sff) * 4 + (E * eff + sff) * 2), like="expert_act_scale")
        up1 = torch.randn(n, E * eff + sff, device=device).to(bf)
        wts = torch.zeros(n, E + 1, device=device)
        wts.scatter_(1, tab[ids.long()].long(), 1.0 / top)
        wts[:, E] = 1.0
        us = timed(lambda: ops.expert_act_scale(up1, wts, E, eff, "relu2"))
        hbm(f"kafepel_expert_act_scale_{label}", us, n * ((top * eff + sff) * 2 + (E * eff + sff) * 2))


def _tenotar_kernels(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device) -> None:
    """The Tenotar design's own kernels, alone, at the preset's sizes: one request of 2,048 prompt tokens, and 8 decoding
    requests of 2,048 cached tokens; beside each the like kernel of the Nudodra design (the closest one the engine has; for
    attention through latents the Nurolorn design's form) at the same sizes.  Attention's arithmetic counts the (query, key)
    pairs that the mask leaves; a decode step's bytes are the cached rows that it leaves."""
    bf = torch.bfloat16
    A = next(x["mixer"] for x in design["layers"] if x["type"] == "attention")
    B = next(x["mixer"] for x in design["layers"] if x["type"] == "attention_2")
    L = next(x["mixer"] for x in design["layers"] if x["type"] == "latent_attention")
    moe = next(x["mlp"] for x in design["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe")
    width = design["width"]
    H, KV, D, V = A["heads"], A["kv_heads"], A["dim"], A["vdim"]
    window, keep, chunk, taps = A["mask"]["size"], A["mask"].get("keep_first", 0), B["mask"]["size"], B["conv"]

    def seen(qs, cs, kind):
        """(query, key) pairs of a step under a mask."""
        total = 0
        for q, c in zip(qs, cs):
            for p in range(c - q, c):
                if kind == "window":
                    lo = max(0, p - window + 1)
                    total += p - lo + 1 + min(keep, lo)
                elif kind == "latent":
                    total += min(p + 1, L["mask"]["size"])
                elif kind == "blocks":
                    total += p % chunk + 1
                else:
                    total += p + 1
        return total

    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n = ctx.num_tokens
        prefill = label.startswith("prefill")
        pool = torch.randn(pages, 2, KV, 16, max(D, V), device=device).to(bf)
        q = (torch.randn(n, H * D, device=device) * 0.3).to(bf)
        slopes = 2.0 ** (-8.0 * torch.arange(1, H + 1, device=device) / H)
        kw = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=A["scale"])

        def attention(name, kind, like=None, **more):
            pairs = seen(qs, cs, kind)
            us = timed(lambda: ops.paged_softmax_attention(q, pool, table, ctx, **kw, **more))
            work = 2.0 * pairs * H * (D + V) if prefill else pairs * KV * (D + V) * 2 + n * H * (D + V) * 2
            (tensor if prefill else hbm)(f"{name}_{label}", us, work, like=like)

        attention("window_keep_first_attention", "window", like="sink_attention", window=window, keep_first=keep)
        attention("block_cap_bias_attention", "blocks", like="sink_attention", chunk=chunk, softcap=B.get("softcap"), slopes=slopes)
        attention("nudodra_sink_attention", "all", sinks=torch.zeros(H, device=device))
        # the heads' preparation: biases, norms, neighbouring lanes, values mixed with an earlier layer's; Nudodra's beside it
        proj = torch.randn(n, (H + KV) * D + KV * V, device=device)
        freq = torch.rand(A["rot"]["dims"] // 2, device=device)
        b_in, qw, kw_ = torch.randn((H + KV) * D + KV * V, device=device), torch.ones(D, device=device), torch.ones(D, device=device)
        first = torch.randn(n, KV * V, device=device)
        us = timed(lambda: ops.head_prepare(proj, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, bias=b_in, q_weight=qw, k_weight=kw_,
                                            eps=1e-6, freq=freq, interleaved=True, values_first=first, values_lambda=0.4, pool=pool, slot_map=slots))
        hbm(f"head_prepare_mixed_values_{label}", us, n * (((H + KV) * D + 2 * KV * V) * 4 + ((H + KV) * D + KV * V) * 2), like="head_prepare")
        us = timed(lambda: ops.head_prepare(proj, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, bias=b_in[: (H + KV) * D], q_weight=qw,
                                            k_weight=kw_, eps=1e-6, freq=freq, values_are_keys=True, pool=pool, slot_map=slots))
        hbm(f"nudodra_head_prepare_{label}", us, n * ((H + KV) * D * 4 + (H + 2 * KV) * D * 2))
        # the short convolution over q, k and v (a streaming kernel: its like is the head norm with a gate, of the same traffic per element)
        C = (H + KV) * D + KV * V
        wc = torch.randn(C, taps, device=device)
        states, sl = torch.zeros(8, taps - 1, C, device=device), i32(list(range(len(qs))))
        us = timed(lambda: ops.short_conv(proj, wc, states, sl, ctx, channels=C))
        hbm(f"short_conv_{label}", us, n * C * 8 + 2 * len(qs) * (taps - 1) * C * 4, like="head_norm_gate")
        o, g2, wn = torch.randn(n, H, V, device=device), torch.randn(n, H * V, device=device), torch.ones(V, device=device)
        us = timed(lambda: ops.head_norm_gate(o, g2, 1e-6, "silu", bf, weight=wn))
        hbm(f"nudodra_head_norm_gate_{label}", us, n * H * V * (4 + 4 + 2))
        # attention through latents: the query latent's norm, the preparation with queries of their own, attention over the cached rows
        LH, rank, rot, hd, qr = L["heads"], L["kv_rank"], L["rot_dim"], L["dim"], L["q_rank"]
        lproj = torch.randn(n, qr + rank + rot + LH, device=device).to(bf)
        wq = torch.ones(qr, device=device)
        us = timed(lambda: ops.row_rmsnorm(lproj[:, :qr], wq, 1e-6))
        hbm(f"row_rmsnorm_{label}", us, n * qr * 4, like="rmsnorm")
        resid, wd = torch.randn(n, width, device=device), torch.ones(width, device=device)
        us = timed(lambda: ops.rmsnorm(resid, wd, 1e-6, out_dtype=bf))
        hbm(f"nudodra_rmsnorm_{label}", us, n * width * 6)
        plane = torch.randn(pages, 16, rank + rot, device=device).to(bf)
        lq = torch.randn(n, LH * (hd + rot), device=device).to(bf)
        lw, lf = torch.ones(rank, device=device), torch.rand(L["rot"]["dims"] // 2, device=device)
        us = timed(lambda: ops.latent_prepare(lproj, ctx.positions, slots, plane, lw, lf, 1e-6, LH, hd, rot, rank, queries=lq, kv_col=qr, halves=True))
        hbm(f"latent_prepare_{label}", us, n * (LH * rot * 4 + (rank + rot) * 4), like="latent_prepare (the Nurolorn design's form)")
        stacked = torch.randn(n, LH * (hd + rot) + rank + rot, device=device).to(bf)
        us = timed(lambda: ops.latent_prepare(stacked, ctx.positions, slots, plane, lw, lf, 1e-6, LH, hd, rot, rank))
        hbm(f"nurolorn_latent_prepare_{label}", us, n * (LH * rot * 4 + (rank + rot) * 4))
        q_lat, q_rot = torch.randn(n, LH, rank, device=device).to(bf), torch.randn(n, LH, rot, device=device).to(bf)
        pairs = seen(qs, cs, "latent")
        for name, win, count in (("latent_window_attention", L["mask"]["size"], pairs), ("nurolorn_latent_attention", None, seen(qs, cs, "all"))):
            us = timed(lambda: ops.latent_paged_attention(q_lat, q_rot, plane, table, ctx, rank=rank, scale=L["scale"], window=win))
            work = 2.0 * count * LH * (2 * rank + rot) if prefill else count * (rank + rot) * 2 + n * LH * (2 * rank + rot) * 2
            (tensor if prefill else hbm)(f"{name}_{label}", us, work, like=None if win is None else "latent attention without a window (the Nurolorn design's)")
        heads_out, gates = torch.randn(n, LH, L["vdim"], device=device).to(bf), torch.randn(n, LH, device=device).to(bf)
        us = timed(lambda: ops.gate_mul(heads_out, gates, "sigmoid", per_head=True))
        hbm(f"gate_a_head_{label}", us, n * LH * L["vdim"] * 4, like="gate_mul (the same kernel with a gate a lane)")
        wide_gates = torch.randn(n, LH * L["vdim"], device=device).to(bf)
        us = timed(lambda: ops.gate_mul(heads_out, wide_gates, "sigmoid"))
        hbm(f"nurolorn_gate_mul_{label}", us, n * LH * L["vdim"] * 6)
        # the router with its bias and the experts' activation with the router's weights, beside Nudodra's with the table's
        E, top, eff, sff = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
        x = torch.randn(n, width, device=device).to(bf)
        wr, br = torch.randn(E, width, device=device) * 0.1, torch.randn(E, device=device)
        us = timed(lambda: ops.route(x, wr, None, E, top, 1.0, True, False, bias=br, shared_one=True))
        hbm(f"router_with_bias_{label}", us, n * width * 2 + E * width * 4 + n * (E + 1) * 4, like="router (the Kafepel design's: the same kernel)")
        corr = torch.zeros(E, device=device)
        us = timed(lambda: ops.route(x, wr, corr, E, top, 2.5, False, False))
        hbm(f"kafepel_router_{label}", us, n * width * 2 + E * width * 4 + n * E * 4)
        up2 = torch.randn(n, 2 * (E * eff + sff), device=device).to(bf)
        wts = ops.route(x, wr, None, E, top, 1.0, True, False, bias=br, shared_one=True)
        us = timed(lambda: ops.expert_gated_act(up2, E, eff, sff, float("inf"), float("inf"), 1.0, weights=wts, up_shift=0.0))
        hbm(f"expert_gated_act_router_weights_{label}", us, n * ((top * eff + sff) * 4 + (E * eff + sff) * 2), like="expert_gated_act")
        tab = torch.rand(design["vocab"], E, device=device).argsort(dim=1)[:, :top].to(torch.int32).contiguous()
        ids = torch.randint(0, design["vocab"], (n,), device=device, dtype=torch.int32)
        us = timed(lambda: ops.expert_gated_act(up2, E, eff, sff, 7.0, 7.0, 1.702, ids=ids, table=tab))
        hbm(f"nudodra_expert_gated_act_{label}", us, n * ((top * eff + sff) * 4 + (E * eff + sff) * 2))


def _zifuzen_kernels(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device) -> None:
    """The Zifuzen design's own kernels, alone, at the preset's sizes: one request of 2,048 prompt tokens, and 8 decoding requests of
    2,048 cached tokens; beside each the like kernel of the Nudodra design (the closest one the engine has), or of the design that
    has one, at the same sizes."""
    bf = torch.bfloat16
    R, A = (next(x["mixer"] for x in design["layers"] if x["type"] == kind) for kind in ("delta", "attention"))
    moe = next(x["mlp"] for x in design["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe")
    dense_ff = next(x["mlp"]["ff"] for x in design["layers"] if x["mlp"] and x["mlp"]["kind"] == "dense")
    width = design["width"]
    H, KV, D, V = A["heads"], A["kv_heads"], A["dim"], A["vdim"]
    RH, RG, RD, RV = R["heads"], R["kv_heads"], R["dim"], R["vdim"]
    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n = ctx.num_tokens
        pairs = sum(q * c - q * (q - 1) // 2 for q, c in zip(qs, cs))
        prefill = label.startswith("prefill")
        sl = i32(list(range(len(qs))))
        # the recurrence with its step sizes, decays, unit vectors, head norm and gate, beside Nudodra's scan and head norm
        C = 2 * RG * RD + RH * RV
        y, proj = torch.randn(n, C, device=device), torch.randn(n, RH * RV + 2 * RH, device=device)
        states = torch.zeros(8, RH, RD, RV, device=device)
        a_log, dt, wn = torch.zeros(RH, device=device), torch.full((RH,), -2.0, device=device), torch.ones(RV, device=device)
        state_bytes = 2 * len(qs) * RH * RD * RV * 4
        us = timed(lambda: ops.delta_rule(y, proj[:, RH * RV : RH * RV + RH], proj[:, RH * RV + RH :], a_log, dt, proj[:, : RH * RV], wn, 1e-6, states, sl,
                                          ctx, heads=RH, kv_heads=RG, dim=RD, value_dim=RV, out_dtype=bf))
        hbm(f"delta_rule_with_norm_and_gate_{label}", us, n * (2 * RG * RD + RH * (2 * RV + 2)) * 4 + n * RH * RV * 2 + state_bytes, like="gated_scan + head_norm_gate")
        rq, rk, rz = (torch.randn(n, RH * RD, device=device) for _ in range(3))
        rv, zb = torch.randn(n, RH * RV, device=device), torch.full((RH * RD,), 3.0, device=device)

        def nudodra_scan():
            o = ops.gated_scan(rq, rk, rv, rz, zb, 0.125, RD ** -0.5, states, sl, ctx.cu_tokens, len(qs), RH, RD, RV, max(qs))
            ops.head_norm_gate(o, proj[:, : RH * RV], 1e-6, "silu", bf, weight=wn)

        us = timed(nudodra_scan)
        hbm(f"nudodra_gated_scan_with_norm_and_gate_{label}", us, n * RH * (3 * RD + 2 * RV) * 4 + n * RH * RV * 2 + state_bytes)
        # the convolution with silu behind it beside Tenotar's without
        u, w = torch.randn(n, C, device=device), torch.randn(C, R["conv"], device=device)
        rows = torch.zeros(8, R["conv"] - 1, C, device=device)
        for name, act in (("short_conv_silu", "silu"), ("tenotar_short_conv", None)):
            us = timed(lambda: ops.short_conv(u, w, rows, sl, ctx, activation=act))
            hbm(f"{name}_{label}", us, n * C * 8, like="short_conv" if act else None)
        # the norm behind a part with the sum and the copy beside the norm in front of one with the sum
        stream, delta, part = (torch.randn(n, width, device=device) for _ in range(3))
        wd = torch.ones(width, device=device)
        us = timed(lambda: ops.post_norm_add(stream, part, wd, 1e-6, copy_dtype=bf))
        hbm(f"post_norm_add_{label}", us, n * width * 14, like="rmsnorm with the sum")
        us = timed(lambda: ops.rmsnorm(stream, wd, 1e-6, delta=delta, out_dtype=bf))
        hbm(f"llama_rmsnorm_with_sum_{label}", us, n * width * 14)
        # attention over all keys, and the heads' preparation
        pool = torch.randn(pages, 2, KV, 16, max(D, V), device=device).to(bf)
        q = (torch.randn(n, H * D, device=device) * 0.3).to(bf)
        kw = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=A["scale"])
        work = 2.0 * pairs * H * (D + V) if prefill else sum(cs) * KV * (D + V) * 2 + n * H * (D + V) * 2
        us = timed(lambda: ops.paged_softmax_attention(q, pool, table, ctx, **kw))
        (tensor if prefill else hbm)(f"attention_{label}", us, work, like="sink_attention")
        sinks = torch.zeros(H, device=device)
        us = timed(lambda: ops.paged_softmax_attention(q, pool, table, ctx, **kw, sinks=sinks))
        (tensor if prefill else hbm)(f"nudodra_sink_attention_{label}", us, work)
        hp, qw, kw_ = torch.randn(n, (H + KV) * D + KV * V, device=device), torch.ones(D, device=device), torch.ones(D, device=device)
        head_bytes = n * ((H + KV) * D + KV * V) * 6
        us = timed(lambda: ops.head_prepare(hp, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, q_weight=qw, k_weight=kw_, eps=1e-6, pool=pool, slot_map=slots))
        hbm(f"head_prepare_{label}", us, head_bytes, like="head_prepare with rotation and biases")
        freq, b_in = torch.rand(D // 4, device=device), torch.randn((H + KV) * D + KV * V, device=device)
        us = timed(lambda: ops.head_prepare(hp, ctx.positions, heads=H, kv_heads=KV, dim=D, value_dim=V, bias=b_in, q_weight=qw, k_weight=kw_, eps=1e-6,
                                            freq=freq, pool=pool, slot_map=slots))
        hbm(f"nudodra_head_prepare_{label}", us, head_bytes)
        # the router with sigmoid scores and groups, the experts' activation, the dense layer's
        E, top, eff, sff = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
        xb, wr, corr = torch.randn(n, width, device=device).to(bf), torch.randn(E, width, device=device) * 0.02, torch.randn(E, device=device)
        groups = moe["router"]["groups"]
        router_bytes = n * width * 2 + E * width * 4 + n * (E + 1) * 4
        us = timed(lambda: ops.route(xb, wr, corr, E, top, 2.5, True, False, shared_one=True, scores="sigmoid", groups=(groups["count"], groups["keep"])))
        hbm(f"router_with_groups_{label}", us, router_bytes, like="router (the Tenotar design's)")
        us = timed(lambda: ops.route(xb, wr, None, E, top, 1.0, True, False, bias=corr, shared_one=True))
        hbm(f"tenotar_router_{label}", us, router_bytes)
        up2 = torch.randn(n, 2 * (E * eff + sff), device=device).to(bf)
        wts = ops.route(xb, wr, corr, E, top, 2.5, True, False, shared_one=True, scores="sigmoid", groups=(groups["count"], groups["keep"]))
        act_bytes = n * ((top * eff + sff) * 4 + (E * eff + sff) * 2)
        us = timed(lambda: ops.expert_gated_act(up2, E, eff, sff, 7.0, 7.0, 1.702, weights=wts))
        hbm(f"expert_gated_act_{label}", us, act_bytes, like="expert_gated_act with the table's weights")
        tab = torch.rand(design["vocab"], E, device=device).argsort(dim=1)[:, :top].to(torch.int32).contiguous()
        ids = torch.randint(0, design["vocab"], (n,), device=device, dtype=torch.int32)
        us = timed(lambda: ops.expert_gated_act(up2, E, eff, sff, 7.0, 7.0, 1.702, ids=ids, table=tab))
        hbm(f"nudodra_expert_gated_act_{label}", us, act_bytes)
        gu, gb = torch.randn(n, 2 * dense_ff, device=device).to(bf), torch.randn(2 * dense_ff, device=device).to(bf)
        for name, act in (("gelu_gate", "gelu_tanh"), ("tenotar_silu_gate", "silu")):
            us = timed(lambda: ops.swiglu(gu, gb, act))
            hbm(f"{name}_{label}", us, n * dense_ff * 6, like="swiglu with biases" if act != "silu" else None)
        # the embedding with positions, the logits' cap
        emb, pos = torch.randn(design["vocab"], width, device=device).to(bf), torch.randn(design["max_positions"], width, device=device).to(bf)
        us = timed(lambda: ops.embed_positions(ids, emb, ctx.positions, pos, 2.0, copy_dtype=bf))
        hbm(f"embed_positions_{label}", us, n * width * 10, like="embed")
        us = timed(lambda: ops.embed(ids, emb))
        hbm(f"llama_embed_{label}", us, n * width * 6)
        if not prefill:
            z = torch.randn(n, design["vocab"], device=device)
            us = timed(lambda: ops.unary(z, "softcap", 30.0, inplace=True))
            hbm(f"logit_cap_{label}", us, n * design["vocab"] * 8, like="logit scale")
            us = timed(lambda: ops.unary(z, "scale", 1.5, inplace=True))
            hbm(f"logit_scale_{label}", us, n * design["vocab"] * 8)


def _pefedra_kernels(design, twin, ops, torch, timed, ctx_for, i32, hbm, tensor, device) -> None:
    """The Pefedra design's own kernels, alone, at the preset's sizes: one request of 2,048 prompt tokens, and 8 decoding requests of
    2,048 cached tokens; beside each the like kernel of the Tenotar design (the closest one the engine has) at the same sizes.
    Attention's arithmetic counts the (query, key) pairs that the window leaves, two maps' for the heads that have two; a decode
    step's bytes are the cached rows that it leaves."""
    bf = torch.bfloat16
    A = next(x["mixer"] for x in design["layers"] if x["type"] == "attention")
    B = next(x["mixer"] for x in design["layers"] if x["type"] == "attention_2")
    width, ff = design["width"], next(x["mlp"]["ff"] for x in design["layers"] if x.get("mlp"))
    window = A["mask"]["size"]

    def seen(qs, cs):
        return sum(min(p + 1, window) for q, c in zip(qs, cs) for p in range(c - q, c))

    for label, qs, cs in (("prefill_2048", [2048], [2048]), ("decode_8x2048", [1] * 8, [2048] * 8)):
        ctx, table, slots, pages = ctx_for(qs, cs)
        n, prefill, pairs = ctx.num_tokens, label.startswith("prefill"), seen(qs, cs)

        def attention(name, H, KV, D, V, maps, like=None, **more):
            pool = torch.randn(pages, 2, KV, 16, max(maps * D, V), device=device).to(bf)
            q = (torch.randn(n, H * maps * D, device=device) * 0.3).to(bf)
            us = timed(lambda: ops.paged_softmax_attention(q, pool, table, ctx, num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=D ** -0.5,
                                                           window=window, **more))
            work = 2.0 * pairs * H * maps * (D + V) if prefill else pairs * KV * (maps * D + V) * 2 + n * H * (maps * D + V) * 2
            (tensor if prefill else hbm)(f"{name}_{label}", us, work, like=like)

        gate = torch.randn(n, B["heads"], device=device)
        turn = torch.rand(n, B["vdim"] // 2, 2, device=device)
        attention("two_map_attention", A["heads"], A["kv_heads"], A["dim"], A["vdim"], 2, like="tenotar_window_attention",
                  differential=ops.DifferentialMaps(0.5, 1e-6, 0.5))
        attention("turned_value_attention", B["heads"], B["kv_heads"], B["dim"], B["vdim"], 1, like="tenotar_window_attention", turn=turn, gate=gate,
                  gate_per_head=True)
        attention("tenotar_window_attention", B["heads"], B["kv_heads"], B["dim"], B["vdim"], 1, keep_first=16)

        def prepare(name, H, KV, D, V, maps, like=None, **more):
            cols = (H + KV) * maps * D + KV * V
            pool = torch.zeros(pages, 2, KV, 16, max(maps * D, V), device=device, dtype=bf)
            proj, bias = torch.randn(n, cols, device=device), torch.randn(cols, device=device)
            us = timed(lambda: ops.head_prepare(proj, ctx.positions, heads=H * maps, kv_heads=KV * maps, dim=D, value_dim=V, bias=bias, pool=pool,
                                                slot_map=slots, maps=maps, **more))
            hbm(f"{name}_{label}", us, n * cols * 6, like=like)

        qw, kw = torch.ones(B["heads"] * B["dim"], device=device), torch.ones(B["kv_heads"] * B["dim"], device=device)
        prepare("head_prepare_two_maps", A["heads"], A["kv_heads"], A["dim"], A["vdim"], 2, like="tenotar_head_prepare", freq=torch.rand(A["rot"]["dims"] // 2, device=device))
        prepare("head_prepare_turned_values", B["heads"], B["kv_heads"], B["dim"], B["vdim"], 1, like="tenotar_head_prepare", q_weight=qw, k_weight=kw, eps=1e-6,
                norm_whole=True, freq=torch.rand(B["rot"]["dims"] // 2, device=device), value_freq=torch.rand(B["vdim"] // 2, device=device), turn_out=turn)
        prepare("tenotar_head_prepare", B["heads"], B["kv_heads"], B["dim"], B["vdim"], 1, q_weight=qw[: B["dim"]].contiguous(), k_weight=kw[: B["dim"]].contiguous(),
                eps=1e-6, freq=torch.rand(B["dim"] // 2, device=device), interleaved=True)
        # the two norms with the token shift, beside one RMS norm that reads the stream and adds nothing
        x, w1, w2, share = torch.randn(n, width, device=device), torch.ones(width, device=device), torch.ones(width, device=device), torch.rand(width, device=device)
        states, sl = torch.zeros(8, width, device=device), i32(list(range(len(qs))))
        us = timed(lambda: ops.shift_norm(x, w1, 1e-6, w2=w2, shift=share, states=states, ctx=ctx, state_slots=sl, out_dtype=bf))
        hbm(f"shift_norm_{label}", us, n * width * 8 + 2 * len(qs) * width * 4, like="tenotar_rmsnorm (one norm)")
        us = timed(lambda: ops.rmsnorm(x, w1, 1e-6, out_dtype=bf))
        hbm(f"tenotar_rmsnorm_{label}", us, n * width * 6)
        # the feed-forward's first product with gelu (decode: one kernel), beside the gated one with SwiGLU of as many weights
        xb = torch.randn(n, width, device=device).to(bf)
        up = (torch.randn(ff, width, device=device) * width ** -0.5).to(bf)
        rows = torch.empty(n, B["heads"] * B["vdim"] + ff, device=device, dtype=bf)
        into = rows[:, B["heads"] * B["vdim"] :]
        us = timed(lambda: ops.linear_act(xb, up, "gelu", out=into))
        work = (2.0 * n * width * ff) if prefill else (ff * width + n * (width + ff)) * 2
        (tensor if prefill else hbm)(f"up_product_gelu_{label}", us, work, like="tenotar_gate_up_swiglu")
        ff2 = twin["intermediate_size"]
        gu, gb = (torch.randn(2 * ff2, width, device=device) * width ** -0.5).to(bf), torch.zeros(2 * ff2, device=device).to(bf)
        us = timed(lambda: ops.swiglu(ops.linear(xb, gu), gb))
        work = (4.0 * n * width * ff2) if prefill else (2 * ff2 * width + n * (width + ff2)) * 2
        (tensor if prefill else hbm)(f"tenotar_gate_up_swiglu_{label}", us, work)
        if prefill:
            z = torch.randn(n, ff, device=device).to(bf)
            us = timed(lambda: ops.unary(z, "gelu", out=into))
            hbm(f"gelu_{label}", us, n * ff * 4, like="tenotar_swiglu")
            z2 = torch.randn(n, 2 * ff2, device=device).to(bf)
            us = timed(lambda: ops.swiglu(z2, gb))
            hbm(f"tenotar_swiglu_{label}", us, n * ff2 * 6)
        # the joined output product into the stream, beside the two products that a pre-norm layer runs
        k1 = B["heads"] * B["vdim"]
        wj = (torch.randn(width, k1 + ff, device=device) * (k1 + ff) ** -0.5).to(bf)
        wo, wd = wj[:, :k1].contiguous(), wj[:, k1 : k1 + ff2].contiguous()
        act = torch.randn(n, k1 + ff, device=device).to(bf)
        sink = ops.ResidualSink(x, None, 0.0)
        us = timed(lambda: sink.linear(act, wj))
        work = (2.0 * n * width * (k1 + ff)) if prefill else ((k1 + ff) * width + n * (k1 + ff)) * 2 + n * width * 8
        (tensor if prefill else hbm)(f"joined_output_product_{label}", us, work, like="tenotar_output_and_down_products")
        a1, a2 = act[:, :k1].contiguous(), act[:, k1 : k1 + ff2].contiguous()
        us = timed(lambda: (sink.linear(a1, wo), sink.linear(a2, wd)))
        work = (2.0 * n * width * (k1 + ff2)) if prefill else ((k1 + ff2) * width + n * (k1 + ff2)) * 2 + n * width * 16
        (tensor if prefill else hbm)(f"tenotar_output_and_down_products_{label}", us, work)


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=200)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", choices=["ours", "reference"], default="ours")
    ap.add_argument("--config", choices=["tinyllama-1.1b", "llama2-7b", "llama3-8b"], default=MODEL,
                    help="tinyllama-1.1b: the headline line (decode of 8 requests).  llama2-7b: 32 requests with prompts of 64 to "
                         "2,048 tokens, 128 new tokens each, through LLM.generate.  llama3-8b: requests arriving at random under a "
                         "fixed number of pages, with preemption")
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the configuration has (recorded in config)")
    ap.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64, the end-to-end run and the kernel table")
    ap.add_argument("--design", choices=["nurolorn-small", "nurolorn-1b", "kafepel-small", "kafepel-1b", "nudodra-small", "nudodra-1b", "tenotar-small",
                                         "tenotar-1b", "pefedra-small", "pefedra-1b", "zifuzen-small", "zifuzen-1b"], default=None,
                    help="instead of the one line: prefill and decode throughput of a Nurolorn, Kafepel, Nudodra, Tenotar, Pefedra or Zifuzen configuration beside a Llama of "
                         "equal width, depth and feed-forward size, and the design's own kernels against their rooflines")
    ap.add_argument("--sweep", action="store_true",
                    help="instead of the one line: a table of decode steps over batch sizes and context lengths and of prefills over prompt lengths")
    args = ap.parse_args()
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not built")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.impl == "reference":
        return reference_arm(args)
    if args.design:
        return design_comparison(args)

    import random

    import torch

    from llmserve_triton_kernels_b200 import LLM, SamplingParams, ops
    from llmserve_triton_kernels_b200.config.presets import PRESETS
    from llmserve_triton_kernels_b200.engine.batch import StepEntry

    peaks, peaks_from = load_peaks()
    cfg_dict = dict(PRESETS[args.config])
    full_layers = cfg_dict["num_hidden_layers"]
    if args.layers:
        cfg_dict["num_hidden_layers"] = args.layers
    device = "cuda:0"
    steps, warmup = args.steps, args.warmup
    page_size = 16
    headline = args.config == MODEL
    prompt_len = PROMPT_LEN if headline else 1024
    batches = (1, 8, 64) if headline else (32,)
    # the K steps are timed several times over (the region of K steps is short against the clock sampler's period); a
    # request decodes through all of them, so the regions are as many as its context allows, 0.3 s of them at most
    room = cfg_dict["max_position_embeddings"] - prompt_len - warmup - 8
    if room < steps:
        print(f"bench.py: {prompt_len} prompt tokens + {warmup + steps} new tokens exceed the context of {cfg_dict['max_position_embeddings']}")
        return 2

    def tokens_for(batch: int, length, seed: int):
        g = torch.Generator().manual_seed(seed)
        lengths = [length] * batch if isinstance(length, int) else length
        return [torch.randint(0, cfg_dict["vocab_size"], (n,), generator=g).tolist() for n in lengths]

    most_batch = max(batches)
    context_pages = -(-((1536 if args.sweep else prompt_len) + room + 64) // page_size)
    llm = LLM(cfg_dict, dtype="bfloat16", device=device, seed=0, block_size=page_size,
              num_blocks=most_batch * context_pages + 256, max_batch_size=most_batch, max_num_batched_tokens=8192)
    cfg = llm.config
    numbers = model_numbers(cfg)
    weight_bytes = llm.model.weight_bytes()
    flush = torch.empty(256 * 2**20, dtype=torch.uint8, device=device)  # larger than the 126 MB L2
    sched = llm.scheduler

    def decode_run(batch: int, k: int, w: int, prompt_len: int = prompt_len, regions: int | None = None) -> dict:
        """``batch`` requests are added to the engine's scheduler and stepped: their prompts first (untimed), then w
        warm-up decode steps, then regions of exactly k decode steps each, every region between synchronisations and
        CUDA events.  One call of ``Scheduler.step()`` launches one decode step (a step's tokens feed the next step on
        the device; the host reads every step's tokens through pinned memory, one step late, inside the region)."""
        sched.reset()
        llm.cache.reset()
        sched.max_batch_size = batch
        new_tokens = cfg.max_position_embeddings - prompt_len - 2
        for prompt in tokens_for(batch, prompt_len, seed=1):
            sched.add_request(prompt, SamplingParams(max_new_tokens=new_tokens))
        guard = 0
        while sched.waiting or any(r.num_computed < len(r.prompt_ids) for r in sched.running):
            sched.step()
            guard += 1
            assert guard < 10000, "the prompts never finished"
        gc.collect()  # the prefill left garbage behind; a full collection (tens of ms) must not fall into the timed steps
        for _ in range(w):
            sched.step()
        torch.cuda.synchronize()
        if regions is None:
            est = 1.0e-3 * k
            regions = max(1, min((new_tokens - w - 16) // k, int(0.3 / est) or 1, 25))
        times, launches0 = [], ops.launch_count()
        first_context = prompt_len + 1 + w
        with ClockSampler() as clocks:
            time.sleep(0.3)  # nvidia-smi is up and sampling before the first region starts
            clocks.begin()
            for _ in range(regions):
                flush.fill_(1)  # L2 holds nothing of the model when a region starts (and 2.2 GB of weights pass through it every step)
                start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                start.record()
                for _ in range(k):
                    sched.step()
                end.record()
                torch.cuda.synchronize()
                times.append(start.elapsed_time(end))
            clocks.end()
        launches = ops.launch_count() - launches0
        assert len(sched.running) == batch and sched.run_ahead, "a request left the batch inside the timed steps"
        ms = statistics.median(times)
        context = first_context + (regions * k) / 2.0  # mean number of cached tokens a timed step reads per request
        bytes_per_step = weight_bytes + batch * context * numbers["kv_bytes_per_token"]
        out = {
            "tokens_per_s": batch * k / (ms / 1e3), "ms_per_step": ms / k, "bytes_per_step": bytes_per_step,
            "gbs": bytes_per_step / (ms / k / 1e3) / 1e9, "launches": launches // regions, "regions": regions,
            "ms_per_step_min": min(times) / k, "ms_per_step_max": max(times) / k,
            "clocks": clocks.summary(), "h2d": llm.step_function.h2d_bytes, "d2h": llm.sampler.d2h_bytes,
        }
        sched.reset()
        return out

    def prefill_run(n_tokens: int = PREFILL_TOKENS) -> dict:
        sched.reset()
        llm.cache.reset()
        prompt = tokens_for(1, n_tokens, seed=2)[0]
        times = []
        for i in range(3 + 5):
            flush.fill_(1)
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            start.record()
            logits = llm.step_function([StepEntry("p", prompt, [n_tokens - 1])])
            ops.argmax(logits)
            end.record()
            torch.cuda.synchronize()
            llm.cache.free_request("p")
            if i >= 3:
                times.append(start.elapsed_time(end))
        ms = statistics.median(times)
        flops = prefill_flops(cfg, n_tokens)
        return {"value": n_tokens / (ms / 1e3), "tokens": n_tokens, "ms": ms,
                "frac": flops / (ms / 1e3) / (peaks["bf16_tflops"] * 1e12), "tflops": flops / (ms / 1e3) / 1e12}

    def e2e_run(batch: int, prompt_lens=None, new_tokens: int = NEW_TOKENS) -> dict:
        """Through ``LLM.generate``: host token ids in, host token ids out.  Run twice; the second run is reported
        (a server meets its shapes again and again: the first meeting of a shape captures its graph)."""
        sched.reset()
        llm.cache.reset()
        sched.max_batch_size = batch
        prompts = tokens_for(batch, prompt_lens or prompt_len, seed=3)
        outs = None
        for _ in range(2):
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            outs = llm.generate(prompts, SamplingParams(max_new_tokens=new_tokens))
            wall = time.perf_counter() - t0
        first = max(o.ttft_s for o in outs)
        last = max(o.total_s for o in outs)
        decoded = sum(len(o.token_ids) - 1 for o in outs)
        ttfts = sorted(o.ttft_s for o in outs)
        return {"value": decoded / (last - first), "unit": "tokens/s", "h2d_bytes_per_step": llm.step_function.h2d_bytes,
                "d2h_bytes_per_step": llm.sampler.d2h_bytes, "ttft_ms": first * 1e3, "ttft_p50_ms": ttfts[len(ttfts) // 2] * 1e3,
                "new_tokens": new_tokens, "all_tokens_per_s": sum(len(o.token_ids) for o in outs) / wall,
                "prompt_tokens": sum(map(len, prompts)), "wall_s": wall, "preemptions": sum(o.num_preemptions for o in outs)}

    def kernel_table() -> dict:
        """The step's dominant kernels one at a time: each as a captured graph of 24 launches in a row over weights that
        rotate through more than L2 holds (as the reference's kernel benchmark rotates its weights:
        benchmarks/bench_decode_matmul.py:28-45), timed by CUDA events around the replay.  GB/s and TFLOP/s against the
        same peaks as the step."""
        h, inter, H, KV, D, V = cfg.hidden_size, cfg.intermediate_size, cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim, cfg.vocab_size
        table = {}

        def timed(fn, n=24):
            fn(0)
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                for i in range(n):
                    fn(i)
            best = float("inf")
            for _ in range(3):
                flush.fill_(1)
                start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                start.record()
                graph.replay()
                end.record()
                torch.cuda.synchronize()
                best = min(best, start.elapsed_time(end) * 1e3 / n)
            return best

        def rotating(rows, cols):
            copies = max(2, -(-(300 << 20) // (rows * cols * 2)))
            return [(torch.randn(rows, cols, device=device) * 0.02).to(torch.bfloat16) for _ in range(min(copies, 40))]

        def hbm(name, us, nbytes):
            table[name] = {"us": round(us, 2), "GB/s": round(nbytes / us / 1e3, 1), "frac": round(nbytes / us / 1e3 / peaks["hbm_gbs"], 3), "bound": "hbm"}

        def tensor(name, us, flops):
            table[name] = {"us": round(us, 2), "TFLOP/s": round(flops / us / 1e6, 1), "frac": round(flops / us / 1e6 / peaks["bf16_tflops"], 3), "bound": "tensor"}

        m = 8
        x, xa = torch.randn(m, h, device=device).to(torch.bfloat16), torch.randn(m, inter, device=device).to(torch.bfloat16)
        resid, norm_w = torch.randn(m, h, device=device), torch.ones(h, device=device)
        sink = ops.ResidualSink(resid, norm_w, 1e-5)
        positions = torch.arange(m, dtype=torch.int32, device=device)
        rotary = torch.randn(64, D, device=device)
        slots = torch.arange(m, dtype=torch.int32, device=device)
        pool = torch.zeros(4, 2, KV, 16, D, dtype=torch.bfloat16, device=device)
        w = rotating((H + 2 * KV) * D, h)
        hbm("decode_qkv_rope_write_8rows", timed(lambda i: ops.linear_qkv_rope(x, w[i % len(w)], positions, rotary, slots, pool, H, KV, D)), w[0].numel() * 2)
        w = rotating(h, H * D)
        xo = torch.randn(m, H * D, device=device).to(torch.bfloat16)
        hbm("decode_out_proj_residual_8rows", timed(lambda i: sink.linear(xo, w[i % len(w)])), w[0].numel() * 2)
        w = rotating(2 * inter, h)
        hbm("decode_gate_up_swiglu_8rows", timed(lambda i: ops.linear_swiglu(x, w[i % len(w)])), w[0].numel() * 2)
        w = rotating(h, inter)
        hbm("decode_down_residual_8rows", timed(lambda i: sink.linear(xa, w[i % len(w)])), w[0].numel() * 2)
        w = rotating(V, h)
        hbm("decode_lm_head_8rows", timed(lambda i: ops.linear(x, w[i % len(w)], out_dtype=torch.float32), n=6), w[0].numel() * 2)
        del w
        # attention of a decode step: 8 requests of 640 cached keys, a pool large enough that the planes rotate out of L2
        from types import SimpleNamespace

        ctx_len, pages_each = 640, 640 // page_size
        planes = max(2, -(-(300 << 20) // (m * pages_each * 2 * KV * page_size * D * 2)))
        pools = torch.randn(planes, m * pages_each, 2, KV, page_size, D, device=device).to(torch.bfloat16)
        table_t = torch.arange(m * pages_each, dtype=torch.int32, device=device).view(m, pages_each).contiguous()
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)  # noqa: E731
        actx = SimpleNamespace(cu_tokens=i32(list(range(m + 1))), context_lens=i32([ctx_len] * m), token_request=i32(list(range(m))),
                               host_cu_tokens=list(range(m + 1)), max_context_len=ctx_len)
        q = torch.randn(m, (H + 2 * KV) * D, device=device).to(torch.bfloat16)
        us = timed(lambda i: ops.paged_attention(q, pools[i % planes], table_t, actx, num_heads=H, num_kv_heads=KV, head_dim=D, scale=D**-0.5))
        hbm("decode_attention_8x640keys", us, m * ctx_len * 2 * KV * D * 2)
        del pools
        # prompt portions of 2,048 tokens: the gated product on the own tcgen05 kernel, the attention on tcgen05
        t = PREFILL_TOKENS
        xp = torch.randn(t, h, device=device).to(torch.bfloat16)
        w = rotating(2 * inter, h)
        tensor("prefill_gate_up_swiglu_2048rows", timed(lambda i: ops.linear_swiglu(xp, w[i % len(w)]), n=8), 2.0 * t * 2 * inter * h)
        del w
        pages_each = t // page_size
        pool1 = torch.randn(pages_each, 2, KV, page_size, D, device=device).to(torch.bfloat16)
        table1 = torch.arange(pages_each, dtype=torch.int32, device=device).view(1, pages_each).contiguous()
        pctx = SimpleNamespace(cu_tokens=i32([0, t]), context_lens=i32([t]), token_request=torch.zeros(t, dtype=torch.int32, device=device),
                               host_cu_tokens=[0, t], max_context_len=t)
        qp = torch.randn(t, (H + 2 * KV) * D, device=device).to(torch.bfloat16)
        us = timed(lambda i: ops.paged_attention(qp, pool1, table1, pctx, num_heads=H, num_kv_heads=KV, head_dim=D, scale=D**-0.5), n=8)
        tensor("prefill_attention_causal_2048", us, 4.0 * H * D * t * (t + 1) / 2.0)
        return table

    if args.sweep:
        print(f"decode steps (bf16, {cfg.num_hidden_layers} layers, {steps} steps a region; bytes = weights + cache of the live requests; peak {peaks['hbm_gbs']:.0f} GB/s {peaks_from})")
        print("| requests | cached tokens each | ms/step | tokens/s | GB/s | of peak |")
        print("|---:|---:|---:|---:|---:|---:|")
        for batch in (1, 8, 16, 32, 64):
            for plen in (128, 512, 1536):
                r = decode_run(batch, steps, warmup, plen, regions=3)
                print(f"| {batch} | {plen + warmup}-{plen + warmup + 3 * steps} | {r['ms_per_step']:.3f} | {r['tokens_per_s']:.0f} | {r['gbs']:.0f} | {r['gbs'] / peaks['hbm_gbs']:.2f} |")
        print(f"prefill of one prompt (peak {peaks['bf16_tflops']:.0f} TFLOP/s {peaks_from})")
        print("| tokens | ms | tokens/s | TFLOP/s | of peak |")
        print("|---:|---:|---:|---:|---:|")
        for n_tokens in (128, 512, 1024, 2048):
            r = prefill_run(n_tokens)
            print(f"| {n_tokens} | {r['ms']:.3f} | {r['value']:.0f} | {r['tflops']:.0f} | {r['frac']:.2f} |")
        e = e2e_run(8)
        print(f"through LLM.generate, 8 prompts of {prompt_len} tokens, {NEW_TOKENS} new tokens each: first tokens after {e['ttft_ms']:.1f} ms, "
              f"{e['value']:.0f} decoded tokens/s, {e['all_tokens_per_s']:.0f} generated tokens/s over the whole call")
        return 0

    main_batch = 8 if headline else 32
    main_run = decode_run(main_batch, steps, warmup)
    clocks = main_run["clocks"]
    rejected = [r for r in clocks["reasons"] if r != "sw_power_cap"]
    if rejected:  # measured once more, as the timing rules ask
        main_run = decode_run(main_batch, steps, warmup)
        clocks = main_run["clocks"]
    prefill = prefill_run()
    points, e2e, kernels, workload = {}, None, None, None
    if not args.skip_points:
        if headline:
            points = {"decode_b1": decode_run(1, steps, warmup)["tokens_per_s"], "decode_b64": decode_run(64, steps, warmup)["tokens_per_s"]}
            e2e = e2e_run(8)
            kernels = kernel_table()
        elif args.config == "llama2-7b":
            # the mixed batch: 32 requests with prompts of 64 to 2,048 tokens, 128 new tokens each, all at once
            rng = random.Random(7)
            e2e = e2e_run(32, prompt_lens=[rng.randint(64, 2048) for _ in range(32)], new_tokens=128)
            workload = "32 requests at once, prompts uniform in [64, 2048], 128 new tokens each"
        else:
            # requests arriving at random (exponential gaps, seeded, as the reference's load test draws them:
            # benchmarks/load_test.py:36-47) under a number of pages that cannot hold them all: the newest is put back
            rng = random.Random(11)
            n_req, new = 48, 256
            lens = [rng.randint(128, 8192 - new - 1) for _ in range(n_req)]
            pages = int(0.45 * sum(-(-(n + new) // page_size) for n in lens[:32]))
            del llm
            gc.collect()
            torch.cuda.empty_cache()
            llm = LLM(cfg_dict, dtype="bfloat16", device=device, seed=0, block_size=page_size, num_blocks=pages, max_batch_size=32,
                      max_num_batched_tokens=8192, chunk_size=2048)
            s2 = llm.scheduler
            prompts = tokens_for(n_req, lens, seed=5)
            for _ in range(2):  # the second pass is reported
                s2.reset()
                llm.cache.reset()
                s2.finished.clear()
                gaps = [rng.expovariate(40.0) for _ in range(n_req)]  # 40 requests a second on average
                arrivals = [sum(gaps[: i + 1]) for i in range(n_req)]
                before = s2.stats.preemptions
                t0, nxt, ids = time.perf_counter(), 0, []
                while nxt < n_req or s2.has_unfinished():
                    now = time.perf_counter() - t0
                    while nxt < n_req and arrivals[nxt] <= now:
                        ids.append(s2.add_request(prompts[nxt], SamplingParams(max_new_tokens=new), arrival_time=t0 + arrivals[nxt]))
                        nxt += 1
                    if s2.has_unfinished():
                        s2.step()
                    else:
                        time.sleep(max(0.0, arrivals[nxt] - now))
                wall = time.perf_counter() - t0
                done = [s2.finished[i] for i in ids]
                ttft = sorted(r.token_times[0] - r.arrival_time for r in done)
                gaps_ms = sorted((b - a) * 1e3 for r in done for a, b in zip(r.token_times, r.token_times[1:]))
                e2e = {"value": n_req * new / wall, "unit": "tokens/s", "wall_s": wall, "ttft_p50_ms": ttft[len(ttft) // 2] * 1e3,
                       "ttft_p99_ms": ttft[-1] * 1e3, "itl_p50_ms": gaps_ms[len(gaps_ms) // 2], "itl_p99_ms": gaps_ms[int(len(gaps_ms) * 0.99)],
                       "preemptions": s2.stats.preemptions - before, "pages": pages, "h2d_bytes_per_step": llm.step_function.h2d_bytes,
                       "d2h_bytes_per_step": llm.sampler.d2h_bytes}
            workload = f"{n_req} requests arriving at 40 a second on average, prompts uniform in [128, 7935], {new} new tokens each, {pages} pages of 16 tokens"
    line = {
        "metric": "decode_tokens_per_s", "value": main_run["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps,
        "warmup": warmup, "ms_per_step": main_run["ms_per_step"], "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "ours",
        "config": {
            "model": f"{args.config} sizes, random weights N(0,0.02) seed 0", "global_batch": main_batch, "seq_len": cfg.max_position_embeddings,
            "prompt_len": prompt_len, "new_tokens": NEW_TOKENS, "parallelism": "single GPU", "layers": cfg.num_hidden_layers,
            "layers_of_config": full_layers, "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads,
            "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size,
            "vocab": cfg.vocab_size, "page_size": page_size, "l2": "256 MiB buffer written before each timed region; weights exceed L2",
            "peaks": peaks_from, "regions": main_run["regions"],
            "timing": "median over the regions of K steps each, every region between synchronisations and CUDA events",
        },
        "clocks": clocks,
        "ms_per_step_range": [main_run["ms_per_step_min"], main_run["ms_per_step_max"]],
        "e2e": e2e,
        "gpu_launches": main_run["launches"],
        "prefill": {k: prefill[k] for k in ("value", "tokens", "ms", "frac")},
        "roofline": {"bound": "hbm", "achieved": main_run["gbs"], "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": main_run["gbs"] / peaks["hbm_gbs"], "bytes_per_step": main_run["bytes_per_step"], "of": peaks_from},
        "points": points,
        "kernels": kernels,
        "kernels_library": ops.loaded_library_path(),
    }
    if workload:
        line["workload"] = workload
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
