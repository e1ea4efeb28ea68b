#!/usr/bin/env python3
"""Decode and prefill throughput of the delta_b200 engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--context 4096] [--layers L] [--shape yi-6b|yi-9b|yi-34b]

Default run: the layer sizes of Yi-6B (32 layers, hidden 4096, 32 heads over 4
key-value heads of 128, intermediate 11008, vocabulary 64000), random bfloat16
weights, 8 requests decoding at a context of 4096 tokens.  One step is one decode
step.  It prints ONE JSON line:

  value      decoded tokens per second, device time of the K timed steps (model step
             and sampling, measured with CUDA events around each step)
  e2e        the same through the Python entry point (LMBackend.step), timed over further runs
             of K steps without the per-step synchronisation the device timing needs: every
             step copies its inputs (positions, block tables, sampling parameters, tokens) from
             pinned host memory and reads the new tokens back to the host.  ``value`` is the
             engine as it runs by default: a decode step is launched while the host still reads
             the step before, with its tokens taken from that step's result on the device;
             ``value_tokens_fed_back_through_host`` is the same with that switched off.
             (Run ahead, the loop can come out a little faster than ``value``: the steps of
             ``value`` are timed one by one, each starting on an idle GPU with its copies on the
             critical path, while here the next step's copies queue behind the running step.)
  prefill    one prompt of 2,048 tokens in one step; frac = flops / time / peak
  roofline   bytes a decode step has to read (every weight once, and the cache of the
             live requests) / its time, against the copy bandwidth
  points     decode tokens per second at batch 1 and 64

Peaks come from MEASURED_PEAKS.json beside this file when it is there, else from the
fallback figures of an earlier measurement of a B200.  The engine runs on one GPU
only: for --gpus above 1 it says so and exits with 2.

Other workloads (``--workload``), each printing one JSON line of the same shape:

  baseline     2,048-token prompts and 512 generated tokens each through ``run_scheduler_loop`` at
               batch 1, 8 and 64 (Yi-6B shape): tokens per second = generated tokens / time of the
               decode steps, and the same over the wall clock of the whole loop
  yi9b-long    Yi-1.5-9B shape, 16 requests of 256 + 3,584 tokens, once with the full cache and
               once with DELTA (``--full_cache_layers 2 --subset_cache_size 64``); both rates and
               their ratio
  yi34b-mixed  Yi-34B shape: steps of one 2,048-token prompt portion beside up to 63 decoding
               requests; milliseconds per mixed step, tokens per second of both kinds, and the
               portion's share of the tensor-core peak
  long-prompt  Yi-6B shape, one prompt of 30,000 tokens (``--context``) in portions of 2,048: milliseconds of the
               first and the last portion, of the whole prompt, and of a decode step behind it
  grown        Yi-6B shape, 64 requests (``--batch``) of 64 + 2,400 tokens: nearly every page is taken
               during decoding, a page at a time in turns with the other requests; the last sixth of
               the decode steps, with the pool handing pages out in runs and one by one

  roletar      the Roletar design (32-bit mixed residual streams, selective scan, latent attention, windowed
               attention with sinks; random weights at widths ``--width``, layers of real sizes) beside the Yi
               architecture at the same width and number of layer runs: prefill of one 2,048-token prompt and
               decode at batch 8, context 2,048, through ``ModelRunner.step``; then every launcher's share of
               one such step with the fraction of the peaks that the elementwise and attention kernels reach

  pibalorn     the Pibalorn design (32-bit residual stream, parallel blocks, attention whose values are its keys,
               linear attention with a decay per head, mixtures of experts; random weights at widths ``--width``)
               beside the Yi architecture, measured as the roletar workload is

  mevulix      the Mevulix design (norms on the sublayers' outputs, latent attention with a query latent, attention with
               capped scores and biases by distance, gelu-gated feed-forwards, experts whose weights multiply their input)
               beside Yi, Pibalorn and Roletar, measured as the roletar workload is

  vazunex      the Vazunex design (gated delta rule with a decay per key channel, state-space recurrence with one decay per
               head, windowed latent attention with a sink and an output gate, experts chosen in groups, identity experts)
               beside Yi, Mufalix, Pibalorn and Roletar, measured as the roletar workload is

  burolorn     the Burolorn design (attention over chunks with a sink and a gate per head behind short convolutions, values mixed
               across layers, token inputs from a second table, experts in groups ranked by two scores) beside Yi, Pibalorn,
               Mevulix and Vazunex, measured as the roletar workload is

``--impl reference`` runs the unmodified hoenza/DELTA engine (baseline/reference_arm.py) on the
default workload and prints its line.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

YI_6B = dict(architectures=["LlamaForCausalLM"], model_type="llama", hidden_size=4096, num_hidden_layers=32,
             num_attention_heads=32, num_key_value_heads=4, intermediate_size=11008, vocab_size=64000,
             rope_theta=5000000.0, rms_norm_eps=1e-5, max_position_embeddings=4096, hidden_act="silu",
             tie_word_embeddings=False, torch_dtype="bfloat16")
# other shapes of the same architecture, for runs beside the default one (--shape)
SHAPES = {
    "yi-6b": ("Yi-6B shape", YI_6B),
    "yi-9b": ("Yi-1.5-9B shape", dict(YI_6B, num_hidden_layers=48, rms_norm_eps=1e-6)),
    "yi-34b": ("Yi-34B shape", dict(YI_6B, hidden_size=7168, num_hidden_layers=60, num_attention_heads=56,
                                    num_key_value_heads=8, intermediate_size=20480)),
}
FALLBACK_PEAKS = dict(hbm_gbs=6650.0, bf16_tflops=1590.0, source="fallback")


def peaks() -> dict:
    p = ROOT / "MEASURED_PEAKS.json"
    if p.is_file():
        try:
            d = json.loads(p.read_text())
            out = dict(hbm_gbs=float(d["hbm_gbs"]), bf16_tflops=float(d["bf16_tflops"]),
                       source="measured")
            return out
        except Exception:  # noqa: BLE001
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self) -> dict:
        if self.proc is None:
            return dict(sm_mhz=None, sm_max_mhz=None, reasons=["nvidia-smi unavailable"])
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        mhz, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for r in self.rows:
            if len(r) < 6:
                continue
            try:
                mhz.append(float(r[0]))
                mx = float(r[1])
            except ValueError:
                continue
            for n, v in zip(names, r[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        mhz.sort()
        return dict(sm_mhz=mhz[len(mhz) // 2] if mhz else None, sm_max_mhz=mx, reasons=sorted(reasons), samples=len(mhz))


def model_numbers(cfg: dict, layers: int):
    d, H, KV = cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"]
    hd = cfg.get("head_dim") or d // H
    I, V = cfg["intermediate_size"], cfg["vocab_size"]
    per_layer = (H + 2 * KV) * hd * d + H * hd * d + 3 * I * d
    weight_bytes = 2 * (layers * (per_layer + 2 * d) + V * d + d)
    kv_bytes_per_token = layers * 2 * KV * hd * 2

    def prefill_flops(T):
        gemm = 2 * T * layers * per_layer + 2 * V * d  # logits for one row
        attn = layers * 4 * hd * H * (T * (T + 1) // 2)
        return gemm + attn
    return weight_bytes, kv_bytes_per_token, prefill_flops


def reference_arm(args) -> int:
    """The unmodified reference on the same decode workload: ``baseline/reference_arm.py`` in a
    process of its own (nothing of delta_b200 is imported there); its JSON line is printed as it
    is.  Whatever goes wrong becomes the ``unavailable`` line with the reason."""
    def unavailable(why: str) -> int:
        print(json.dumps({"impl": "reference", "unavailable": " ".join(why.split())[:400]}))
        return 0
    if args.gpus != 1:
        return unavailable("the reference arm is set up for one GPU")
    script = ROOT / "baseline" / "reference_arm.py"
    if not (ROOT / "baseline" / "_ref" / "DELTA").is_dir():
        return unavailable("no copy of hoenza/DELTA under baseline/_ref (it has no setup.py or pyproject.toml, so pip "
                           "cannot install it; a plain copy of the tree is what its own scripts use)")
    if args.shape == "yi-9b":
        return unavailable("the reference's table of models has no 48-layer Yi entry (DELTA/Engine/DELTA/model.py:72-97)")
    cmd = [sys.executable, str(script), "--batch", str(args.batch), "--context", str(args.context), "--steps", str(args.steps),
           "--warmup", str(max(3, args.warmup)), "--shape", args.shape]
    if args.no_graph:
        cmd.append("--no-graph")
    try:
        r = subprocess.run(cmd, capture_output=True, text=True, timeout=1500)
    except subprocess.TimeoutExpired:
        return unavailable("the reference did not finish within 1500 s")
    sys.stderr.write(r.stderr[-4000:])
    for line in reversed(r.stdout.splitlines()):
        if line.startswith('{"impl"'):
            print(line)
            return 0
    tail = (r.stderr.strip().splitlines() or r.stdout.strip().splitlines() or ["no output"])[-1]
    return unavailable(f"the reference ended with code {r.returncode}: {tail}")


def _flat_config(shape_name, cfg, layers, **more) -> dict:
    d = cfg["hidden_size"]
    out = {"model": shape_name, "layers": layers, "layers_of_named_config": cfg["num_hidden_layers"], "hidden": d,
           "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
           "head_dim": cfg.get("head_dim") or d // cfg["num_attention_heads"], "intermediate": cfg["intermediate_size"],
           "vocab": cfg["vocab_size"], "page_size": 16, "parallelism": "single GPU"}
    out.update(more)
    return out


def _loop(eng, prompts, max_new, timed: bool):
    """Runs the requests through ``run_scheduler_loop``.  Timed: every step between CUDA events
    (returns the decode steps' records); untimed: as a user runs it, wall clock only."""
    import torch
    eng.step_timings.clear()
    eng.record_timings = timed
    eng.add_requests(prompts, [len(p) + max_new for p in prompts], [], max_new_tokens=max_new)
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    eng.run_scheduler_loop()
    wall = time.perf_counter() - t0
    eng.record_timings = False
    decode = [r for r in eng.step_timings if r["tokens"] == r["active_bsz"]]
    return decode, wall


def other_workload(args) -> int:
    import torch
    from delta_b200.engine import LMBackend
    from delta_b200.kernels import ops
    pk = peaks()
    gen = torch.Generator().manual_seed(1)
    name = args.workload
    shape = {"baseline": "yi-6b", "yi9b-long": "yi-9b", "yi34b-mixed": "yi-34b", "grown": "yi-6b", "long-prompt": "yi-6b"}[name]
    shape_name, shape_cfg = SHAPES[shape]
    layers = args.layers or shape_cfg["num_hidden_layers"]
    cfg = dict(shape_cfg, num_hidden_layers=layers)
    weight_bytes, kv_per_tok, prefill_flops = model_numbers(cfg, layers)

    def prompts(n, length):
        return [torch.randint(0, cfg["vocab_size"], (length,), generator=gen).tolist() for _ in range(n)]

    def engine(max_batch, max_len, **kw):
        e = LMBackend(dtype=torch.bfloat16, device="cuda:0", cuda_graph_decode=not args.no_graph)
        e.load_model(config_json=cfg, seed=0)
        e.setup_caches(max_batch_size=max_batch, max_seq_length=max_len, page_size=16, **kw)
        e.scheduler.decode_while_prefill = False
        return e

    clocks = ClockSampler()
    if name == "baseline":
        plen, new = 2048, args.generate or 512
        eng = engine(64, plen + new, max_tokens_per_step=2048)
        points, e2e, ms = {}, {}, {}
        clocks.start()
        for b in (1, 8, 64):
            _loop(eng, prompts(b, plen), 24, True)                     # records the graphs of this batch size
            decode, _ = _loop(eng, prompts(b, plen), new, True)
            full = [r for r in decode if r["active_bsz"] == b]
            t = sum(r["model_forward_ms"] + r["postprocess_ms"] for r in full)
            points[f"decode_b{b}"] = b * len(full) / (t / 1e3)
            ms[f"b{b}"] = t / len(full)
            l0 = ops.launch_count()
            _, wall = _loop(eng, prompts(b, plen), new, False)
            e2e[f"b{b}"] = b * new / wall        # prompts included in the time: what a user of the loop sees
        clk = clocks.stop()
        ctx = plen + new / 2
        achieved = (weight_bytes + 8 * ctx * kv_per_tok) / (ms["b8"] / 1e3) / 1e9
        out = {"workload": name, "metric": f"decode tok/s ({shape_name}, bf16, 2,048-token prompts + {new} generated, batch 1/8/64)",
               "value": points["decode_b8"], "unit": "tokens/s", "n_gpus": 1, "ms_per_step": ms["b8"], "higher_is_better": True,
               "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
               "config": _flat_config(shape_name, shape_cfg, layers, global_batch=8, seq_len=plen + new, prompt_len=plen,
                                      generated=new, cuda_graph_decode=not args.no_graph, peaks=pk["source"]),
               "points": points, "ms_per_decode_step": ms,
               "e2e": {"unit": "generated tokens/s over the wall clock of the whole loop, prompts included", **e2e},
               "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": achieved / pk["hbm_gbs"]},
               "clocks": clk}
    elif name == "yi9b-long":
        B, plen, new = 16, 256, args.generate or 3584
        res = {}
        clocks.start()
        for mode in ("full", "delta"):
            eng = engine(B, plen + new, max_tokens_per_step=4096, enable_selective_cache=mode == "delta",
                         full_cache_layers=[2] if mode == "delta" else None, subset_cache_size=64)
            _loop(eng, prompts(B, plen), 24, True)
            decode, _ = _loop(eng, prompts(B, plen), new, True)
            t = sum(r["model_forward_ms"] + r["postprocess_ms"] for r in decode)
            _, wall = _loop(eng, prompts(B, plen), new, False)
            tail = decode[-max(1, len(decode) // 8):]       # the last eighth: the longest contexts
            res[mode] = dict(tokens_per_s=B * len(decode) / (t / 1e3), ms_per_step=t / len(decode),
                             ms_per_step_last_eighth=sum(r["model_forward_ms"] + r["postprocess_ms"] for r in tail) / len(tail),
                             e2e_tokens_per_s=B * new / wall, steps=len(decode))
            del eng
            torch.cuda.empty_cache()
        clk = clocks.stop()
        out = {"workload": name, "metric": f"decode tok/s ({shape_name}, bf16, batch {B}, {plen}-token prompts + {new} generated)",
               "value": res["delta"]["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "ms_per_step": res["delta"]["ms_per_step"],
               "higher_is_better": True, "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
               "config": _flat_config(shape_name, shape_cfg, layers, global_batch=B, seq_len=plen + new, prompt_len=plen,
                                      generated=new, full_cache_layers="2", subset_cache_size=64, cuda_graph_decode=not args.no_graph),
               "full_cache": res["full"], "delta": res["delta"],
               "delta_over_full": res["delta"]["tokens_per_s"] / res["full"]["tokens_per_s"], "clocks": clk}
    elif name == "long-prompt":
        # One prompt of 30,000 tokens (--context sets another length) in portions of 2,048, then 16 decoded tokens: the
        # portions' attention reads what the portions before left in the cache, so the later ones are bound by it.
        plen = args.context if args.context != 4096 else 30000
        cfg = dict(cfg, max_position_embeddings=max(cfg.get("max_position_embeddings", 0), plen + 64))
        eng = engine(2, plen + 64, max_tokens_per_step=2048)
        clocks.start()
        for _ in range(2):              # the second run is the measured one (kernels chosen, buffers made)
            records, _ = None, None
            eng.step_timings.clear()
            eng.record_timings = True
            eng.add_requests(prompts(1, plen), [plen + 16], [], max_new_tokens=16)
            eng.run_scheduler_loop()
            eng.record_timings = False
            records = list(eng.step_timings)
        clk = clocks.stop()
        pre = [r["model_forward_ms"] + r["postprocess_ms"] for r in records if r["tokens"] > 1]
        dec = [r["model_forward_ms"] + r["postprocess_ms"] for r in records if r["tokens"] == 1]
        flops = prefill_flops(plen)
        out = {"workload": name, "metric": f"prefill tok/s ({shape_name}, bf16, one prompt of {plen} tokens in portions of 2,048)",
               "value": plen / (sum(pre) / 1e3), "unit": "tokens/s", "n_gpus": 1, "ms_per_step": sum(pre) / len(pre), "higher_is_better": True,
               "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
               "config": _flat_config(shape_name, shape_cfg, layers, global_batch=1, seq_len=plen, portion=2048, peaks=pk["source"]),
               "prompt_ms": sum(pre), "first_portion_ms": pre[0], "last_full_portion_ms": pre[-2] if len(pre) > 1 else pre[-1],
               "decode_ms_per_step_at_the_end": sum(dec) / max(1, len(dec)),
               "prefill": {"value": plen / (sum(pre) / 1e3), "tokens": plen, "ms": sum(pre), "frac": flops / (sum(pre) / 1e3) / (pk["bf16_tflops"] * 1e12)},
               "clocks": clk}
    elif name == "grown":
        # Many requests with short prompts that decode for a long time, in turns: nearly every page of a request
        # is taken during decoding, one at a time, between the pages the other requests take.  Measured with the
        # pool handing out runs of pages, and with the one-page last-in-first-out stack.
        B, plen, new = args.batch if args.batch != 8 else 64, 64, args.generate or 2400
        res = {}
        clocks.start()
        for runs in (True, False):
            eng = engine(B, plen + new, max_tokens_per_step=4096, page_runs=runs)
            _loop(eng, prompts(B, plen), 24, True)
            decode, _ = _loop(eng, prompts(B, plen), new, True)
            tail = decode[-max(1, len(decode) // 6):]
            res[runs] = sum(r["model_forward_ms"] + r["postprocess_ms"] for r in tail) / len(tail)
            del eng
            torch.cuda.empty_cache()
        clk = clocks.stop()
        ctx = plen + new * 11 / 12
        achieved = (weight_bytes + B * ctx * kv_per_tok) / (res[True] / 1e3) / 1e9
        out = {"workload": name, "metric": f"decode tok/s ({shape_name}, bf16, batch {B}, {plen}-token prompts + {new} generated, last sixth of the steps)",
               "value": B / (res[True] / 1e3), "unit": "tokens/s", "n_gpus": 1, "ms_per_step": res[True], "higher_is_better": True,
               "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
               "config": _flat_config(shape_name, shape_cfg, layers, global_batch=B, seq_len=plen + new, prompt_len=plen, generated=new,
                                      cuda_graph_decode=not args.no_graph, peaks=pk["source"]),
               "ms_per_step_pages_in_runs": res[True], "ms_per_step_pages_one_by_one": res[False],
               "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": achieved / pk["hbm_gbs"]},
               "clocks": clk}
    else:
        B, portion, ctx_len = 64, 2048, 4096
        eng = engine(B, ctx_len, max_tokens_per_step=portion + B)
        eng.scheduler.decode_while_prefill = True
        n_mixed = max(4, min(args.steps, 12))
        # 63 requests decode from a context of 1,024 tokens on; then one prompt of 2,048 tokens is added per step
        eng.add_requests(prompts(B - 1, 1024), [ctx_len] * (B - 1), [])
        while eng.scheduler.waiting or any(not r.output for r in eng.scheduler.running):
            eng.step()
        for _ in range(4):
            eng.step()
        records = []
        clocks.start()
        eng.record_timings = True
        for k in range(n_mixed + 2):
            eng.add_requests(prompts(1, portion), [portion + 1], [])     # ends after its first token: its slot is free again
            eng.step_timings.clear()
            eng.step()
            records.extend(eng.step_timings)
        eng.record_timings = False
        clk = clocks.stop()
        mixed = [r for r in records if r["tokens"] > portion][2:]
        t = sum(r["model_forward_ms"] + r["postprocess_ms"] for r in mixed) / len(mixed)
        dec = sum(r["active_bsz"] - 1 for r in mixed) / len(mixed)
        out = {"workload": name, "metric": f"mixed step ({shape_name}, bf16): one {portion}-token prompt portion beside {B - 1} decoding requests",
               "value": (portion + dec) / (t / 1e3), "unit": "tokens/s", "n_gpus": 1, "ms_per_step": t, "higher_is_better": True,
               "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
               "config": _flat_config(shape_name, shape_cfg, layers, global_batch=B, seq_len=ctx_len, portion=portion, steps=len(mixed)),
               "prefill_tokens_per_s": portion / (t / 1e3), "decode_tokens_per_s": dec / (t / 1e3),
               "chunk": {"flops": prefill_flops(portion), "frac": prefill_flops(portion) / (t / 1e3) / (pk["bf16_tflops"] * 1e12),
                         "peak_tflops": pk["bf16_tflops"]},
               "weights_gb": weight_bytes / 1e9, "clocks": clk}
    print(json.dumps(out))
    return 0


def roletar_config(d: int) -> dict:
    """A Roletar model with layers of the sizes of a real model of width d: a selective state-space layer, two latent
    attention layers that run twice, a windowed attention layer with sinks; four residual streams."""
    H = d // 128
    ff = dict(kind="dense", ff=4 * d)
    lat = dict(type="latent_attention", mlp=ff, mixer=dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=256, scale=192 ** -0.5,
                                                           rot=dict(base=10000.0, dims=64)))
    return dict(architecture="Roletar", vocab=32000, width=d, streams=4, logit_softcap=30.0, norm=dict(eps=1e-6),
                loop=dict(start=1, stop=3, times=2),
                layers=[dict(type="mamba1", mlp=ff, mixer=dict(inner=2 * d, state=16, conv=4, dt_rank=d // 16)), lat, dict(lat),
                        dict(type="attention", mlp=ff, mixer=dict(heads=H, kv_heads=max(1, H // 4), dim=128, vdim=128, scale=128 ** -0.5,
                                                                 mask=dict(size=1024)))])


def yi_like_config(d: int, layers: int) -> dict:
    """The closest existing model at equal size: as many layer runs, the same width and heads, a SwiGLU of equal weight count."""
    return dict(YI_6B, hidden_size=d, num_hidden_layers=layers, num_attention_heads=d // 128, num_key_value_heads=max(1, d // 512),
                intermediate_size=(8 * d // 3 + 255) // 256 * 256, vocab_size=32000, max_position_embeddings=8192)


def pibalorn_config(d: int) -> dict:
    """A Pibalorn model with layers of the sizes of a real model of width d: a linear-attention layer with a dense gated
    feed-forward, then an attention layer and a linear-attention layer with mixtures of 16 experts (4 chosen, 4d/8 wide each,
    and a shared expert) that run twice, then another attention layer; a pair table of 4,093 buckets."""
    H = d // 128
    lin = dict(type="lightning", mixer=dict(heads=H, dim=128, vdim=128, decay=[1.0 - 2.0 ** (-5 - 3 * h / max(1, H - 1)) for h in range(H)]))
    att = dict(type="attention", mixer=dict(heads=H, kv_heads=max(1, H // 4), dim=128, vdim=128, scale=0.09, rot=dict(base=10000.0, dims=64)))
    experts = dict(kind="moe", router=dict(experts=16, top=4), expert=dict(ff=d // 2, limit=7.0), shared=dict(ff=d // 2, limit=7.0))
    return dict(architecture="Pibalorn", vocab=32000, width=d, norm=dict(eps=1e-5),
                embedding=dict(scale=float(d) ** 0.5, bigram=dict(buckets=4093, mul_prev=8191, mul_cur=131)),
                loop=dict(start=1, stop=3, times=2),
                layers=[dict(lin, mlp=dict(kind="dense", ff=(8 * d // 3 + 255) // 256 * 256, limit=7.0)), dict(att, mlp=experts), dict(lin, mlp=experts),
                        dict(att, mlp=experts)])


def mufalix_config(d: int) -> dict:
    """A Mufalix model with layers of the sizes of a real model of width d: a matrix-memory layer (d/128 heads of 128 x 128), then
    a layer of two mixers side by side (attention of d/128 heads on d/512 key-value heads over a window of 1,024 tokens, 64 of 128
    entries rotated with scaled frequencies; a recurrence of d channels in groups of 128 behind a convolution of 4 taps) and a
    second matrix-memory layer that run twice, then another pair; every layer with a mixture of 16 experts (4 chosen, d/2 wide)."""
    H = d // 128
    mem = dict(type="mlstm", mixer=dict(heads=H, dim=128, vdim=128, gate_cap=15.0))
    pair = dict(type="parallel", mixer=dict(
        left=dict(heads=H, kv_heads=max(1, H // 4), dim=128, vdim=128, scale=0.09, mask=dict(size=1024),
                  rot=dict(base=500000.0, dims=64, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))),
        right=dict(width=d, conv=4, blocks=H)))
    experts = dict(kind="moe", router=dict(experts=16, top=4, scale=2.5), expert=dict(ff=d // 2))
    return dict(architecture="Mufalix", vocab=32000, width=d, norm=dict(eps=1e-5), embedding=dict(scale=float(d) ** 0.5),
                loop=dict(start=1, stop=3, times=2),
                layers=[dict(mem, mlp=experts), dict(pair, mlp=experts), dict(mem, mlp=experts), dict(pair, mlp=experts)])


def mevulix_config(d: int) -> dict:
    """A Mevulix model with layers of the sizes of a real model of width d: latent attention (d/128 heads of 128 plain and 64 rotated
    entries, latents of 256 for keys and values and 3d/8 for queries, ramp-scaled rotary positions) and grouped-query attention
    (d/128 heads on d/512 key-value heads, capped scores, a bias table of 32 rows up to distance 1,024, a query temperature), one
    of the attention layers reading another's keys and values; dense gated feed-forwards and mixtures of 16 experts (4 chosen, d/2
    wide each, and a shared expert) take turns."""
    H = d // 128
    lat = dict(type="latent_attention", mixer=dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=256, q_rank=3 * d // 8, scale=0.07,
                                                   rot=dict(base=500000.0, dims=64, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0))))
    att = dict(heads=H, kv_heads=max(1, H // 4), dim=128, vdim=128, scale=0.09, softcap=50.0, q_temp=dict(coef=0.1, every=512),
               bias_max=1024, bias_rows=32)
    experts = dict(kind="moe", router=dict(experts=16, top=4), expert=dict(ff=d // 2), shared=dict(ff=d // 2))
    dense = dict(kind="dense", ff=(8 * d // 3 + 255) // 256 * 256)
    return dict(architecture="Mevulix", vocab=32000, width=d, norm=dict(eps=1e-5), logit_scale=0.5,
                layers=[dict(lat, mlp=experts), dict(type="attention", mixer=att, mlp=dense), dict(lat, mlp=experts),
                        dict(type="attention", mixer=dict(att, kv_from=1), mlp=experts), dict(lat, mlp=dense),
                        dict(type="attention", mixer=att, mlp=experts)])


def vazunex_config(d: int) -> dict:
    """A Vazunex model with layers of the sizes of a real model of width d: state-space layers (inner width 2 d, d/32 heads of 64, 128
    states, two groups of maps), gated delta rule layers (d/128 heads of 128, ranks of 128), latent attention (d/128 heads of 128 plain
    and 64 rotated entries, a latent of 256, a window of 1,024); every layer with a mixture of 16 experts (4 chosen, d/2 wide each) and
    4 identities in 4 groups of which 2 are kept."""
    H = d // 128
    ssd = dict(type="mamba2", mixer=dict(heads=d // 32, vdim=64, state=128, groups=2, conv=4, norm_groups=1))
    delta = dict(type="channel_delta", mixer=dict(heads=H, kv_heads=H, dim=128, vdim=128, conv=4, decay_rank=128, gate_rank=128))
    lat = dict(type="latent_attention", mixer=dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=256, scale=0.07, mask=dict(size=1024),
                                                   rot=dict(base=500000.0, dims=64)))
    mlp = dict(kind="moe", router=dict(experts=16, top=4, identity=4, groups=dict(count=4, keep=2), scale=2.0), expert=dict(ff=d // 2))
    return dict(architecture="Vazunex", vocab=32000, width=d, norm=dict(eps=1e-5), logit_scale=0.5, residual_mult=0.5,
                layers=[dict(L, mlp=mlp) for L in (ssd, delta, lat, delta, ssd, lat)])


def burolorn_config(d: int) -> dict:
    """A Burolorn model with layers of the sizes of a real model of width d: attention of d/128 heads of 128 on d/512 key-value heads behind
    convolutions of 4 taps, 64 of 128 entries rotated, chunks of 1,024 tokens in two of three layers, values mixed across layers; token
    inputs of 256; dense gated feed-forwards and mixtures of 16 experts (4 chosen, d/2 wide each, and a shared expert; 2 of 4 groups are
    kept) take turns."""
    H = d // 128
    att = dict(heads=H, kv_heads=max(1, H // 4), dim=128, vdim=128, scale=0.09, conv=4, rot=dict(base=500000.0, dims=64), v_mix=True)
    experts = dict(kind="moe", router=dict(experts=16, top=4, groups=dict(count=4, keep=2), scale=2.0), expert=dict(ff=d // 2), shared=dict(ff=d // 2))
    dense = dict(kind="dense", ff=(8 * d // 3 + 255) // 256 * 256)
    return dict(architecture="Burolorn", vocab=32000, width=d, norm=dict(eps=1e-5), logit_scale=0.5, token_side=dict(dim=256),
                layers=[dict(type="attention", mixer=dict(att, mask=dict(size=1024)) if i % 3 < 2 else att, mlp=dense if i % 2 == 0 else experts)
                        for i in range(6)])


def roletar_workload(args) -> int:
    return design_workload(args, "roletar")


def design_workload(args, design: str) -> int:
    """Prefill (one prompt of 2,048 tokens in one step) and decode (batch 8 at context 2,048) of a design (Roletar, Pibalorn, Mufalix, Mevulix, Vazunex, Burolorn) beside the
    Yi architecture at equal width and layer count (Mufalix also beside Pibalorn, the closest design; Mevulix beside Pibalorn and Roletar;
    Vazunex beside Mufalix, Pibalorn and Roletar; Burolorn beside Mevulix, Vazunex and Pibalorn), through ``ModelRunner.step``, timed with CUDA events after warm-up with
    the L2 flushed before every timed step; then every launcher's share of one such step, with the fraction of the measured
    peaks that the design's own kernels and their Yi counterparts reach."""
    import torch
    from delta_b200.config import EngineConfig
    from delta_b200.engine.step import ModelRunner, RowInput
    from delta_b200.kernels import ops
    pk = peaks()
    T, B, CTX = 2048, 8, 2048
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda:0")
    gen = torch.Generator().manual_seed(1)
    clocks = ClockSampler()
    clocks.start()
    Design = design.capitalize()
    out = {"workload": design, "metric": f"prefill tok/s and decode tok/s ({Design} beside Yi at equal width and layer runs, bf16)",
           "unit": "tokens/s", "n_gpus": 1, "higher_is_better": True, "dtype": "bf16", "data": "synthetic token ids, random weights",
           "steps": args.steps, "warmup": args.warmup, "peaks": pk, "sizes": {}}

    def timed(fn, reps):
        ts = []
        for _ in range(reps):
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1))
        ts.sort()
        return ts[len(ts) // 2]

    def measure(cfg_json, vocab):
        ec = EngineConfig(max_batch=B + 1, max_seq_len=CTX + 64, page_size=16, dtype="bfloat16", max_tokens_per_step=T,
                          num_pages=(B + 1) * (CTX + 64) // 16, cuda_graph_decode=True)
        r = ModelRunner(config_json=cfg_json, seed=0, engine_config=ec)
        prompt = torch.randint(0, vocab, (T,), generator=gen).tolist()
        res = {}

        def prefill():
            slot = r.cache.acquire_slot()
            r.run_rows([RowInput(slot, prompt, 0, [T - 1])])
            r.cache.release_slot(slot)
        for _ in range(max(3, args.warmup // 2)):
            prefill()
        res["prefill_ms"] = timed(prefill, max(3, args.steps // 8))
        ops.profile_start()
        prefill()
        res["prefill_launchers"] = ops.profile_stop()
        # decode: B requests at context CTX (filled in portions), then single tokens
        slots = [r.cache.acquire_slot() for _ in range(B)]
        for s in slots:
            r.run_rows([RowInput(s, prompt[:CTX - 8], 0, [])])
        pos = [CTX - 8]

        def decode():
            r.run_rows([RowInput(s, [7], pos[0], [0]) for s in slots])
        for _ in range(3):
            decode()
            pos[0] += 1
        res["decode_ms"] = timed(decode, max(3, args.steps // 8))     # (the same position is run again: equal work)
        ops.profile_start()
        decode()
        res["decode_launchers"] = ops.profile_stop()
        l0 = ops.launch_count()
        decode()
        res["launches_per_decode_step"] = ops.launch_count() - l0
        # the same step replayed from a recorded CUDA graph with sampling, as generation runs it
        for s in slots:
            r.cache.grow(s, pos[0] + 1)

        def decode_graph():
            r.step_and_sample([RowInput(s, [7], pos[0], [0]) for s in slots])
        for _ in range(4):
            decode_graph()
        res["decode_graph_ms"] = timed(decode_graph, max(3, args.steps // 8)) if r.decode_graph_ready(B) else None
        del r
        torch.cuda.empty_cache()
        return res

    launches = 0
    for d in args.width:
        rc = {"roletar": roletar_config, "pibalorn": pibalorn_config, "mufalix": mufalix_config, "mevulix": mevulix_config, "vazunex": vazunex_config,
              "burolorn": burolorn_config}[design](d)
        runs = 6
        yc = yi_like_config(d, runs)
        a, b = measure(rc, rc["vocab"]), measure(yc, yc["vocab_size"])
        if design in ("mufalix", "mevulix", "vazunex", "burolorn"):     # the closest design of the engine (32-bit stream, layer norms, experts beside a shared one) as well
            pc = pibalorn_config(d)
            c = measure(pc, pc["vocab"])
        if design in ("mevulix", "vazunex"):     # and the one whose mixers are the closest (latent attention, attention with a sink over a cache of rows)
            oc = roletar_config(d)
            c2 = measure(oc, oc["vocab"])
        if design == "vazunex":     # recurrent mixers behind a 32-bit stream, gated norms, a windowed attention with a sink and a gate
            mc = mufalix_config(d)
            c3 = measure(mc, mc["vocab"])
        if design == "burolorn":     # attention with a sink, dense layers and mixtures in turn; short convolutions
            ec, zc = mevulix_config(d), vazunex_config(d)
            c4, c5 = measure(ec, ec["vocab"]), measure(zc, zc["vocab"])
        launches += a["launches_per_decode_step"]
        H = d // 128
        # what the kernels of one step have to move or compute, per launcher (prefill of T tokens unless said otherwise)
        S, C, N = 4, 2 * d, 16
        work = {   # launcher: (bytes, flops) of ALL its calls in a prefill step
            "stream_norm": ((2 * S * d * 4 + 2 * d * 2) * T * (2 * runs), 0),
            "selective_scan": ((4 * C + 2 * N) * 2 * T, 0),
            "conv_silu": (2 * C * 2 * T, 0),
            "activation": (2 * 4 * d * 2 * T * runs, 0),
            "latent_prepare": ((H * 192 + 320 + 320 + H * 64) * 2 * T * 4, 0),
            "rows_append": ((H + 2 * max(1, H // 4)) * 128 * 2 * T, 0),
            "gemm_nt_plain_batched": (0, 2 * T * H * (128 * 256 + 256 * 128) * 4),
            "attention_rows_mma": (0, 4 * (2 * H * (320 + 256) * T * (T + 1) // 2)),      # the latent layers; the windowed one:
            "attention_rows_tc": (0, 2 * H * 256 * (1024 * T - 1024 * 1023 // 2)),
        }
        def pibalorn_work():
            G, top, F = max(1, H // 4), 4, d // 2
            n_lin, n_att, n_moe = 3, 3, 5          # runs of a linear-attention layer, of an attention layer, of a mixture
            return {
                "residual_norm": ((2 * d * 4 + 3 * d * 2) * T * runs, 0),
                "embedding_pair": ((2 * d * 2 + 2 * d * 4) * T, 0),
                "glu_clamped": (3 * (((8 * d // 3 + 255) // 256 * 256) + n_moe * F) * 2 * T, 0),
                "rows_append_unit": ((2 * H + 3 * G) * 128 * 2 * T * n_att, 0),
                "gated_rms_norm": ((H * 128 * 4 + 2 * H * 128 * 2) * T * n_lin, 0),
                "experts_combine": ((top * d * 4 + 2 * d * 2) * T * n_moe, 0),
                "decay_attention_chunked": (0, 2 * T * H * (2 * 128 * 128 + 16 * (128 + 128)) * n_lin),
                "experts_gemm_tc": (0, 2 * T * top * 3 * d * F * n_moe),
                "attention_rows_tc": (0, 4 * 128 * H * (T * (T + 1) // 2) * n_att),
            }
        if design == "pibalorn":
            work = pibalorn_work()

        def mufalix_work():
            G, top, F, Wn = max(1, H // 4), 4, d // 2, 1024
            n_mem, n_pair, n_moe = 3, 3, 6          # runs of a matrix-memory layer, of a pair of mixers, of a mixture
            seen = Wn * T - Wn * (Wn - 1) // 2       # (query, key) pairs inside the window
            return {
                "residual_norm": ((2 * d * 4 + 2 * d * 4 + d * 2) * T * (2 * runs), 0),
                "matrix_memory_chunked": (0, 2 * T * H * (2 * 128 * 128 + 16 * (128 + 128)) * n_mem),     # counted as the linear attention's
                "gated_rms_norm": ((H * 128 * 4 + 2 * H * 128 * 2) * T * (n_mem + n_pair), 0),
                "gated_recurrence": ((2 * d * 4 + 3 * d * 2) * T * n_pair, 0),
                "conv_silu": (2 * d * 2 * T * n_pair, 0),
                "normed_sum": (3 * d * 4 * T * n_pair, 0),
                "rows_append_unit": ((2 * H + 4 * G) * 128 * 2 * T * n_pair, 0),
                "sigmoid_gate": (3 * H * 128 * 2 * T * n_pair, 0),
                "activation": (2 * top * F * 2 * T * n_moe, 0),
                "experts_combine": ((top * d * 4 + d * 4) * T * n_moe, 0),
                "experts_gemm_tc": (0, 2 * T * top * 2 * d * F * n_moe),
                "attention_rows_tc": (0, 4 * 128 * H * seen * n_pair),
            }
        if design == "mufalix":
            work = mufalix_work()

        def vazunex_work():
            top, F, Hs, P, Ns, G, Wn = 4, d // 2, d // 32, 64, 128, 2, 1024
            n_ssd, n_delta, n_lat, n_moe = 2, 2, 2, 6
            ch = Hs * P + 2 * G * Ns                  # channels of a state-space layer's convolution
            seen = Wn * T - Wn * (Wn - 1) // 2
            real = 16 / 20                           # the share of the choices that are experts, when the choices are spread evenly
            return {
                "residual_norm": ((2 * d * 4 + 3 * d * 2) * T * (2 * runs), 0),
                "embedding_pair": ((d * 2 + d * 4) * T, 0),
                "conv_silu": ((2 * ch * n_ssd + 2 * 3 * d * n_delta) * 2 * T, 0),
                "state_space_chunked": (0, 2 * T * Hs * (2 * Ns * P + 16 * P) * n_ssd + 2 * T * G * 16 * Ns * n_ssd),
                "delta_rule_chunked": (0, 2 * T * H * (3 * 128 * 128 + 16 * (2 * 128 + 128)) * n_delta),
                "gated_rms_norm": ((Hs * P * (4 + 2 + 2) * n_ssd + H * 128 * (4 + 4 + 2) * n_delta) * T, 0),
                "latent_prepare": ((H * 192 + 320 + 320 + H * 64) * 2 * T * n_lat, 0),
                "sigmoid_gate": (3 * H * 128 * 2 * T * n_lat, 0),
                "experts_gather": (2 * top * real * d * 2 * T * n_moe, 0),
                "experts_combine": ((top * real * d * 4 + d * 2 + d * 4) * T * n_moe, 0),
                "experts_gemm_tc": (0, 2 * T * top * real * 3 * d * F * n_moe),
                "library batched product": (0, 2 * T * H * (128 * 256 + 256 * 128) * n_lat),
                "gemm_nt_plain_batched": (0, 2 * T * H * (128 * 256 + 256 * 128) * n_lat),
                "attention_rows_mma": (0, 2 * H * (320 + 256) * seen * n_lat),
            }
        if design == "vazunex":
            work = vazunex_work()

        def mevulix_work():
            G, top, F, Fd, Rq = max(1, H // 4), 4, d // 2, (8 * d // 3 + 255) // 256 * 256, 3 * d // 8
            n_lat, n_att, n_own, n_moe, n_dense = 3, 3, 2, 4, 2      # latent layers, attention layers, of which with keys of their own, mixtures, dense
            pairs = T * (T + 1) // 2
            return {
                "sublayer_norm_add": ((2 * d * 4 + 2 * d * 2) * T * (2 * runs), 0),
                "residual_norm": ((d * 4 + d * 2) * T, 0),
                "rms_norm_strided": (2 * Rq * 2 * T * n_lat, 0),
                "latent_prepare": ((H * 192 + 320 + 320 + H * 64) * 2 * T * n_lat, 0),      # counted as in the Roletar table: the whole query row
                "rows_append_unit": (((2 * H + 4 * G) * n_own + 2 * H * (n_att - n_own)) * 128 * 2 * T, 0),
                "glu_clamped": (3 * (Fd * n_dense + F * n_moe) * 2 * T, 0),
                "experts_scale_rows": ((1 + top) * d * 2 * T * n_moe, 0),
                "experts_gather": (2 * top * d * 2 * T * n_moe, 0),
                "experts_combine": ((top * d * 4 + 2 * d * 2) * T * n_moe, 0),
                "experts_gemm_tc": (0, 2 * T * top * 3 * d * F * n_moe),
                "library batched product": (0, 2 * T * H * (128 * 256 + 256 * 128) * n_lat),
                "gemm_nt_plain_batched": (0, 2 * T * H * (128 * 256 + 256 * 128) * n_lat),
                "attention_rows_mma": (0, 2 * H * (320 + 256) * pairs * n_lat + 4 * 128 * H * pairs * n_att),
            }
        if design == "mevulix":
            work = mevulix_work()
        if design == "burolorn":
            G, top, F, Fd, n, Cn = max(1, H // 4), 4, d // 2, (8 * d // 3 + 255) // 256 * 256, 256, 1024
            n_att, n_full, n_moe, n_dense = 6, 2, 3, 3
            ch = (H + 2 * G) * 128                     # channels of a layer's convolutions
            chunks = T // Cn * (Cn * (Cn + 1) // 2)      # (query, key) pairs inside the chunks
            work = {
                # per layer: two sums with a norm behind them (one of a sublayer's output, one of the token input), one that leaves the stream rounded
                "residual_norm": ((3 * (2 * d * 4 + 2 * d * 2)) * T * runs, 0),
                "embedding_pair": ((d * 2 + d * 4) * T, 0),
                "rows_conv_append": ((2 * ch + G * 128) * 2 * T * n_att, 0),      # in, out, and the values that are mixed
                "table_gate": (3 * n * 2 * T * runs, 0),
                "glu_clamped": (3 * (Fd * n_dense + F * n_moe) * 2 * T, 0),
                "experts_gather": (2 * top * d * 2 * T * n_moe, 0),
                "experts_combine": ((top * d * 4 + 2 * d * 2) * T * n_moe, 0),
                "experts_gemm_tc": (0, 2 * T * top * 3 * d * F * n_moe),
                "attention_rows_tc": (0, 4 * 128 * H * (chunks * (n_att - n_full) + T * (T + 1) // 2 * n_full)),
            }
        roletar_work = {
            "stream_norm": ((2 * S * d * 4 + 2 * d * 2) * T * (2 * runs), 0),
            "latent_prepare": ((H * 192 + 320 + 320 + H * 64) * 2 * T * 4, 0),
            "rows_append": ((H + 2 * max(1, H // 4)) * 128 * 2 * T, 0),
            "gemm_nt_plain_batched": (0, 2 * T * H * (128 * 256 + 256 * 128) * 4),
            "library batched product": (0, 2 * T * H * (128 * 256 + 256 * 128) * 4),
            "attention_rows_mma": (0, 4 * (2 * H * (320 + 256) * T * (T + 1) // 2)),      # the latent layers; the windowed one:
            "attention_rows_tc": (0, 2 * H * 256 * (1024 * T - 1024 * 1023 // 2)),
            "selective_scan": ((4 * C + 2 * N) * 2 * T, 0),
            "conv_silu": (2 * C * 2 * T, 0),
        }
        yi_work = {
            "rms_norm": (4 * d * 2 * T * (2 * runs) , 0),
            "silu_mul": (3 * yc["intermediate_size"] * 2 * T * runs, 0),
            "rope_append": ((H + 2 * max(1, d // 512)) * 128 * 2 * 2 * T * runs, 0),
            "attention_prefill_tc": (0, 4 * 128 * H * (T * (T + 1) // 2) * runs),
        }

        def fractions(launchers, table):
            rows = {}
            for name, (calls, ms) in sorted(launchers.items(), key=lambda kv: -kv[1][1]):
                row = {"calls": calls, "ms": round(ms, 4)}
                if name in table and ms > 0:
                    by, fl = table[name]
                    if by:
                        row["gbs"] = round(by / ms / 1e6, 1)
                        row["of_measured_copy"] = round(by / ms / 1e6 / pk["hbm_gbs"], 3)
                    if fl:
                        row["tflops"] = round(fl / ms / 1e9, 1)
                        row["of_measured_bf16"] = round(fl / ms / 1e9 / pk["bf16_tflops"], 3)
                rows[name] = row
            return rows
        out["sizes"][str(d)] = {
            design: {"prefill_tok_s": T / a["prefill_ms"] * 1e3, "prefill_ms": a["prefill_ms"], "decode_tok_s": B / a["decode_ms"] * 1e3,
                        "decode_ms": a["decode_ms"], "decode_graph_ms": a["decode_graph_ms"], "launches_per_decode_step": a["launches_per_decode_step"],
                        "prefill_launchers": fractions(a["prefill_launchers"], work),
                        "decode_launchers": fractions(a["decode_launchers"], {})},
            "yi": {"prefill_tok_s": T / b["prefill_ms"] * 1e3, "prefill_ms": b["prefill_ms"], "decode_tok_s": B / b["decode_ms"] * 1e3,
                   "decode_ms": b["decode_ms"], "decode_graph_ms": b["decode_graph_ms"], "launches_per_decode_step": b["launches_per_decode_step"],
                   "prefill_launchers": fractions(b["prefill_launchers"], yi_work),
                   "decode_launchers": fractions(b["decode_launchers"], {})},
            **({"pibalorn": {"prefill_tok_s": T / c["prefill_ms"] * 1e3, "prefill_ms": c["prefill_ms"], "decode_tok_s": B / c["decode_ms"] * 1e3,
                             "decode_ms": c["decode_ms"], "decode_graph_ms": c["decode_graph_ms"],
                             "launches_per_decode_step": c["launches_per_decode_step"],
                             "prefill_launchers": fractions(c["prefill_launchers"], pibalorn_work()),
                             "decode_launchers": fractions(c["decode_launchers"], {})}} if design in ("mufalix", "mevulix", "vazunex", "burolorn") else {}),
            **({"mufalix": {"prefill_tok_s": T / c3["prefill_ms"] * 1e3, "prefill_ms": c3["prefill_ms"], "decode_tok_s": B / c3["decode_ms"] * 1e3,
                            "decode_ms": c3["decode_ms"], "decode_graph_ms": c3["decode_graph_ms"],
                            "launches_per_decode_step": c3["launches_per_decode_step"],
                            "prefill_launchers": fractions(c3["prefill_launchers"], mufalix_work()),
                            "decode_launchers": fractions(c3["decode_launchers"], {})}} if design == "vazunex" else {}),
            **({"roletar": {"prefill_tok_s": T / c2["prefill_ms"] * 1e3, "prefill_ms": c2["prefill_ms"], "decode_tok_s": B / c2["decode_ms"] * 1e3,
                            "decode_ms": c2["decode_ms"], "decode_graph_ms": c2["decode_graph_ms"],
                            "launches_per_decode_step": c2["launches_per_decode_step"],
                            "prefill_launchers": fractions(c2["prefill_launchers"], roletar_work),
                            "decode_launchers": fractions(c2["decode_launchers"], {})}} if design in ("mevulix", "vazunex") else {}),
            **({name: {"prefill_tok_s": T / m["prefill_ms"] * 1e3, "prefill_ms": m["prefill_ms"], "decode_tok_s": B / m["decode_ms"] * 1e3,
                       "decode_ms": m["decode_ms"], "decode_graph_ms": m["decode_graph_ms"], "launches_per_decode_step": m["launches_per_decode_step"],
                       "prefill_launchers": fractions(m["prefill_launchers"], table), "decode_launchers": fractions(m["decode_launchers"], {})}
                for name, m, table in (("mevulix", c4, mevulix_work()), ("vazunex", c5, vazunex_work()))} if design == "burolorn" else {}),
            "config": {"width": d, "layer_runs": runs, "prefill_tokens": T, "decode_batch": B, "decode_context": CTX,
                       "l2": "flushed before every timed step"}}
    first = out["sizes"][str(args.width[0])]
    out.update(value=first[design]["prefill_tok_s"], ms_per_step=first[design]["prefill_ms"], vs_baseline=None,
               gpu_launches=launches, clocks=clocks.stop(),
               config={"model": f"{Design}, width {args.width[0]}, 6 layer runs", "global_batch": 1, "seq_len": T, "parallelism": "single GPU"})
    print(json.dumps(out))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the shape has (both numbers go into config)")
    ap.add_argument("--shape", choices=sorted(SHAPES), default="yi-6b")
    ap.add_argument("--impl", default="ours")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--skip-points", action="store_true")
    ap.add_argument("--enable_selective_cache", action="store_true", help="DELTA on (not the default run)")
    ap.add_argument("--full_cache_layers", nargs="+", type=int, default=[0, 1, 2, 14, 22])
    ap.add_argument("--subset_cache_size", type=int, default=64)
    ap.add_argument("--workload", choices=["decode", "baseline", "yi9b-long", "yi34b-mixed", "grown", "long-prompt", "roletar", "pibalorn", "mufalix", "mevulix", "vazunex", "burolorn"],
                    default="decode")
    ap.add_argument("--width", type=int, nargs="+", default=[2048, 4096], help="--workload roletar / pibalorn / mufalix / mevulix / vazunex / burolorn: the model widths that are measured")
    ap.add_argument("--generate", type=int, default=None, help="tokens generated per request in the other workloads (default: what the workload names)")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm(args)
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported (single-GPU engine tier)")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.workload in ("roletar", "pibalorn", "mufalix", "mevulix", "vazunex", "burolorn"):
        return design_workload(args, args.workload)
    if args.workload != "decode":
        return other_workload(args)

    import torch
    from delta_b200.engine import LMBackend
    from delta_b200.kernels import ops

    shape_name, shape_cfg = SHAPES[args.shape]
    full_layers = shape_cfg["num_hidden_layers"]
    if args.layers is None:
        args.layers = full_layers
    cfg = dict(shape_cfg, num_hidden_layers=args.layers)
    pk = peaks()
    weight_bytes, kv_per_tok, prefill_flops = model_numbers(cfg, args.layers)
    ctx_len = args.context
    max_b = 64 if not args.skip_points else args.batch
    eng = LMBackend(dtype=torch.bfloat16, device="cuda:0", cuda_graph_decode=not args.no_graph)
    eng.load_model(config_json=cfg, seed=0)
    eng.setup_caches(max_batch_size=max(max_b, args.batch), max_seq_length=ctx_len, page_size=16, max_tokens_per_step=2048,
                     enable_selective_cache=args.enable_selective_cache,
                     full_cache_layers=args.full_cache_layers if args.enable_selective_cache else None,
                     subset_cache_size=args.subset_cache_size)
    gen = torch.Generator().manual_seed(1)

    def fresh_prompts(n, length):
        return [torch.randint(0, cfg["vocab_size"], (length,), generator=gen).tolist() for _ in range(n)]

    def run_decode(batch, steps, warmup, through_api_wall=False):
        """Prefills ``batch`` requests so that the timed decode steps end at the context
        length, then times ``steps`` decode steps.  Returns (device ms per step, end-to-end
        ms per step, launches per step, bytes in, bytes out, mean context)."""
        total_new = warmup + 3 * steps + 3
        plen = ctx_len - total_new
        sch = eng.scheduler
        sch.decode_while_prefill = False
        eng.add_requests(fresh_prompts(batch, plen), [ctx_len] * batch, [])
        while sch.waiting or any(not r.output for r in sch.running):
            eng.step()
        for _ in range(warmup):
            eng.step()
        torch.cuda.synchronize()
        l0 = ops.launch_count()
        dev_ms = 0.0
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        eng.record_timings = True
        eng.step_timings.clear()
        for _ in range(steps):
            eng.step()
        torch.cuda.synchronize()
        eng.record_timings = False
        dev_ms = sum(s["model_forward_ms"] + s["postprocess_ms"] for s in eng.step_timings) / steps
        launches = (ops.launch_count() - l0) / steps
        mean_ctx = plen + warmup + steps / 2
        # the same number of steps again as a user drives them: no per-step synchronisation for
        # timing, so the engine launches each decode step while the host still reads the one before
        e2e = []
        for ahead in (False, True):     # tokens fed back through the host; then on the device, one step ahead
            eng.run_ahead = ahead
            eng.step()
            torch.cuda.synchronize()
            e0.record()
            for _ in range(steps):
                eng.step()
            e1.record()
            torch.cuda.synchronize()
            e2e.append(e0.elapsed_time(e1) / steps)
        e2e_ms = tuple(e2e)
        h2d = eng.runner.last_staging_bytes
        sch.abort_all("bench")
        return dev_ms, e2e_ms, launches, h2d, 4 * batch, mean_ctx

    # ---- prefill of 2,048 tokens ------------------------------------------------
    T = 2048
    pre_ms = []
    for i in range(3):
        eng.add_requests(fresh_prompts(1, T), [T + 1], [])
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        eng.step()
        e1.record()
        torch.cuda.synchronize()
        pre_ms.append(e0.elapsed_time(e1))
        eng.scheduler.abort_all("bench")
    pre = min(pre_ms[1:])
    prefill = dict(value=T / (pre / 1e3), tokens=T, ms=pre, frac=prefill_flops(T) / (pre / 1e3) / (pk["bf16_tflops"] * 1e12))

    # ---- the headline: decode at the default batch --------------------------------
    clocks = ClockSampler()
    clocks.start()
    dev_ms, e2e_ms, launches, h2d, d2h, mean_ctx = run_decode(args.batch, args.steps, args.warmup)
    clk = clocks.stop()
    value = args.batch / (dev_ms / 1e3)
    bytes_step = weight_bytes + args.batch * mean_ctx * kv_per_tok
    achieved = bytes_step / (dev_ms / 1e3) / 1e9
    points = {}
    if not args.skip_points:
        for b in (1, 64):
            d_ms, _, _, _, _, _ = run_decode(b, max(16, args.steps // 2), args.warmup)
            points[f"decode_b{b}"] = b / (d_ms / 1e3)

    out = {
        "metric": f"decode tok/s ({shape_name}, bf16, batch {args.batch}, context {ctx_len})", "value": value, "unit": "tokens/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": dev_ms, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights N(0,0.02), random token ids)",
        "config": _flat_config(shape_name, shape_cfg, args.layers, global_batch=args.batch, seq_len=ctx_len,
                               cuda_graph_decode=not args.no_graph, selective_cache=bool(args.enable_selective_cache),
                               l2="inputs larger than L2 (weights %.1f GB)" % (weight_bytes / 1e9), peaks=pk["source"]),
        "e2e": {"value": args.batch / (e2e_ms[1] / 1e3), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h,
                "value_tokens_fed_back_through_host": args.batch / (e2e_ms[0] / 1e3)},
        "gpu_launches": int(round(launches * args.steps)),
        "clocks": clk,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": achieved / pk["hbm_gbs"]},
        "points": points,
    }
    from delta_b200.parts import linear
    print("kernels chosen per product (rows bucket, N, K, swiglu, out): " +
          "; ".join(f"{k[0]}x{k[1]}x{k[2]}{'sw' if k[3] else ''}->{v}" for k, v in sorted(linear.choices().items(), key=str)),
          file=sys.stderr)
    print("measured in isolation, us:",
          "; ".join(f"{k[0]}x{k[1]}x{k[2]}{'sw' if k[3] else ''}: " + " ".join(f"{c}={t:.1f}" for c, t in v.items())
                    for k, v in sorted(linear.timings().items(), key=str)), file=sys.stderr)
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
