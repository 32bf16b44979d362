#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at Qwen3-8B sizes with random weights, on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--batch B]
    python bench.py --workload 14b-mixed | 32b-long          (the two further measured workloads, one line each)

Prints ONE JSON line.  ``value`` is decoded tokens per second at batch 8 (a "step" is one
decode step of the whole batch, timed on the device with CUDA events); ``e2e`` is the
same through the Python entry point with host token ids in and out every step;
``prefill`` is one 2,048-token prompt; ``roofline`` relates the decode step's bytes
(every weight it uses once plus the cache of the live requests) to the HBM peak;
``points`` holds decode at batch 1 and 64 (``points_roofline``: each point's time per step
and fraction of the HBM peak).  Peaks come from MEASURED_PEAKS.json beside this file when
present, else from the fallback figures of this pool.

``--marginal``: instead of the benchmark line, what each kernel family costs INSIDE the captured decode step (batch
``--batch``, prompts of ``--prompt-len`` tokens): the step is timed whole and again with that family's launches left out
(the results are then wrong, only the clock is read).  The difference is what the family adds to the step with all the
overlap between neighbouring kernels that programmatic dependent launch gives, which a kernel timed alone cannot show.
``--marginal-prefill``: the same for the step that runs one whole prompt of ``--prompt-len`` tokens.

``--workload 14b-mixed``: Qwen3-14B layer sizes, 32 requests with prompts of 128 to 4,096
random tokens, all present at the start, run by the engine's scheduler with portions of 512
prompt tokens beside the decoding requests' tokens, 256 tokens each at temperature 0.7,
context 8,192: total tokens per second, time to first token, and what the steps held.
``--workload 32b-long``: Qwen3-32B layer sizes, 8 requests with 12,000-token prompts, then 256
greedy tokens each, context 16,384: decode tokens per second, its fraction of the HBM peak,
and the share of the step that is spent on the long cache (against the same step at 16 keys).

The reference (a Rust crate) cannot be installed here: ``--impl reference`` says so.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# layer sizes of the benchmark configuration (Qwen3-8B)
QWEN3_8B = {
    "architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "vocab_size": 151936, "hidden_size": 4096,
    "num_hidden_layers": 36, "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128,
    "intermediate_size": 12288, "rms_norm_eps": 1e-6, "rope_theta": 1000000.0, "max_position_embeddings": 40960,
    "tie_word_embeddings": False, "use_sliding_window": False, "torch_dtype": "bfloat16",
}
QWEN3_14B = dict(QWEN3_8B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408)
QWEN3_32B = dict(QWEN3_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600)
CONTEXT = 4096          # tokens per request the cache is sized for
PROMPT = 2048           # tokens each request holds before decoding is timed


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed regions run."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                          "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
        sm = sorted(int(r[0]) for r in self.rows if r and r[0].isdigit())
        mx = [int(r[1]) for r in self.rows if len(r) > 1 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 2 + i and r[2 + i] == "Active" for r in self.rows)]
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None, "reasons": reasons,
                "samples": len(sm)}


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=0, help="run this many of the configuration's layers (0 = all)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    ap.add_argument("--workload", default="headline", choices=["headline", "14b-mixed", "32b-long", "lokinex", "tabedra", "kupelix", "kozasun", "sefelorn", "gemodra"])
    ap.add_argument("--sizes", default="1024,2048", help="with --workload lokinex, tabedra, kupelix, kozasun, sefelorn or gemodra: widths to run")
    ap.add_argument("--marginal", action="store_true", help="marginal cost of each kernel family inside the decode step")
    ap.add_argument("--prompt-len", type=int, default=PROMPT, help="with --marginal: tokens each request holds")
    ap.add_argument("--marginal-prefill", action="store_true",
                    help="marginal cost of each kernel family inside the step that runs one whole prompt of --prompt-len tokens")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "the reference is a Rust crate (no setup.py/pyproject.toml; "
                          "no cargo or rustc in this image): pip cannot install it"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.marginal_prefill:
        return marginal_costs_prefill(args)
    if args.marginal:
        return marginal_costs(args)
    if args.workload == "14b-mixed":
        return mixed_workload(args)
    if args.workload == "32b-long":
        return long_context_workload(args)
    if args.workload == "lokinex":
        return lokinex_workload(args)
    if args.workload in ("tabedra", "kupelix", "kozasun", "sefelorn", "gemodra"):
        return lokinex_workload(args, design=args.workload)

    import numpy as np
    import torch
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.engine import roofline
    from rustingstrata_b200.sampling import SamplingParams

    pk = roofline.peaks(os.path.join(ROOT, "MEASURED_PEAKS.json"))
    cfg = dict(QWEN3_8B)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    n_layers = cfg["num_hidden_layers"]
    max_batch = max(args.batch, 1 if args.no_points else 64)
    eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=max_batch * CONTEXT,
                 max_batch_tokens=PROMPT, max_seqs=max_batch)
    runner = eng.runner
    rng = np.random.default_rng(0)
    V = cfg["vocab_size"]
    wbytes = roofline.weight_bytes(runner.model)
    clocks = ClockSampler()

    def prefill_requests(n):
        """Admits n requests and runs their 2,048-token prompts, one prompt per step."""
        rids = []
        for _ in range(n):
            rids.append(eng.add_request(rng.integers(0, V, size=PROMPT).tolist(), CONTEXT - PROMPT, SamplingParams()))
        while eng.scheduler.waiting or any(r.prefilling for r in eng.scheduler.running):
            eng.step()
        return rids

    def finish_all():
        eng.drain()
        for r in list(eng.scheduler.running):
            eng.scheduler.running.remove(r)
            runner.release(r.rid)
            eng._samplers.pop(r.rid, None)

    def time_decode(n, steps, warmup):
        """Device-timed decode of n requests; returns (ms per step, e2e ms per step, launches per step, kv tokens)."""
        prefill_requests(n)
        for _ in range(warmup):
            eng.step()
        kv_tokens = sum(runner.length(r.rid) for r in eng.scheduler.running)
        # kernels of this package that run inside the timed region: its steps are graph replays, whose kernel nodes the
        # runner counted at capture (the warm-up steps of the device-timed loop, launched from Python, are not timed)
        ms = eng.decode_steps_device_timed(steps, warmup=3)
        launches = eng.kernels_in_timed_steps / steps
        # end to end through Engine.step: every step's inputs go up from pinned host memory and its chosen ids come
        # back to the host.  The engine launches a step while the one before it still runs, so the region starts and
        # ends with nothing under way: `steps` calls, then the step the last call launched ahead is taken in too.
        eng.drain()
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        for _ in range(steps):
            eng.step()
        done_steps = steps + (1 if eng._flight is not None else 0)
        eng.drain()
        torch.cuda.synchronize()
        e2e_ms = (time.perf_counter() - t0) * 1000 / done_steps
        finish_all()
        return ms, e2e_ms, launches, kv_tokens

    # ---- prefill of one 2,048-token prompt (warm-up runs first)
    for _ in range(2):
        prefill_requests(1)
        finish_all()
    clocks.start()
    torch.cuda.synchronize()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    rid_prompt = rng.integers(0, V, size=PROMPT).tolist()
    eng.add_request(rid_prompt, CONTEXT - PROMPT, SamplingParams())
    eng.lookahead = False                      # the timed step is the prompt alone, not the first decode step behind it
    ev0.record()
    eng.step()
    ev1.record()
    eng.lookahead = True
    torch.cuda.synchronize()
    prefill_ms = ev0.elapsed_time(ev1)
    finish_all()
    pf_flops = roofline.step_flops(runner.model, [PROMPT], [PROMPT], 1)
    prefill = {"value": PROMPT / prefill_ms * 1000, "tokens": PROMPT, "ms": prefill_ms,
               "frac": pf_flops / (prefill_ms / 1000) / (pk["bf16_tflops"] * 1e12)}

    # ---- decode at the headline batch
    ms, e2e_ms, launches, kv_tokens = time_decode(args.batch, args.steps, args.warmup)
    points, points_roofline = {}, {}
    if not args.no_points:
        for b in (1, 64):
            pms, _, _, pkv = time_decode(b, max(64, args.steps), args.warmup)
            points[f"decode_b{b}"] = b / pms * 1000
            pr = roofline.decode_roofline(runner.model, runner.kv_bytes_per_token, pkv, pms, pk)
            points_roofline[f"decode_b{b}"] = {"ms_per_step": pms, "steps": max(64, args.steps), "achieved": pr["achieved"],
                                               "frac": pr["frac"]}
    clk = clocks.stop()

    step_bytes = wbytes + kv_tokens * runner.kv_bytes_per_token
    achieved = step_bytes / (ms / 1000) / 1e9
    value = args.batch / ms * 1000
    rec = {
        "metric": "decode tok/s at batch 8 (Qwen3-8B sizes, bf16, random weights, 2,048-token prompts)",
        "value": value, "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "ms_per_step": ms,
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"model": "qwen3-8b-sizes", "layers": n_layers, "layers_of_config": full_layers,
                   "hidden": cfg["hidden_size"], "q_heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate": cfg["intermediate_size"], "vocab": V, "global_batch": args.batch,
                   "seq_len": CONTEXT, "prompt_len": PROMPT, "page_size": 16, "parallelism": "single-gpu",
                   "weights": "random N(0,0.02) bf16", "l2": "inputs larger than L2 (weights + cache)",
                   "peaks": pk["source"]},
        "e2e": {"value": args.batch / e2e_ms * 1000, "unit": "tok/s", "h2d_bytes_per_step": eng.h2d_bytes_last_step,
                "d2h_bytes_per_step": eng.d2h_bytes_last_step},
        "gpu_launches": int(round(launches * args.steps)),
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": achieved / pk["hbm_gbs"]},
        "points": points,
        "points_roofline": points_roofline,
        "clocks": clk,
    }
    print(json.dumps(rec))
    return 0


def marginal_costs(args) -> int:
    """Times the captured decode step whole, then with one kernel family's launches left out at a time."""
    import numpy as np
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.kernels import ops
    from rustingstrata_b200.sampling import SamplingParams
    cfg = dict(QWEN3_8B)
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    L, B, S = cfg["num_hidden_layers"], args.batch, args.prompt_len
    eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=B * CONTEXT, max_batch_tokens=PROMPT, max_seqs=B)
    rng = np.random.default_rng(0)
    for _ in range(B):
        eng.add_request(rng.integers(0, cfg["vocab_size"], size=S).tolist(), CONTEXT - S, SamplingParams())
    while eng.scheduler.waiting or any(r.prefilling for r in eng.scheduler.running):
        eng.step()

    def timed():
        eng.runner._graphs.clear()                       # the step is captured anew, without the launches that are off
        return eng.decode_steps_device_timed(max(args.steps, 32), warmup=4)
    for _ in range(3):
        timed()                                          # until the clocks have settled under the power cap
    whole = timed()
    out = {"batch": B, "prompt_len": S, "layers": L, "ms_per_step": whole, "us_per_layer": whole / L * 1000, "marginal_us_per_layer": {},
           "marginal_us_per_step": {}}
    H, I = cfg["hidden_size"], cfg["intermediate_size"]
    qkv = (cfg["num_attention_heads"] + 2 * cfg["num_key_value_heads"]) * cfg["head_dim"]
    families = [("attention_decode (+ merge)", "attention_decode", None), ("qk_norm_rope_kv", "qk_norm_rope_kv", None),
                ("gate/up product", "linear_swiglu", None), ("row norms (+ owed sums)", "rmsnorm", None),
                ("qkv product", "linear", (qkv, H)), ("output product", "linear", (H, cfg["num_attention_heads"] * cfg["head_dim"])),
                ("down product", "linear", (H, I)), ("output head", "linear", (cfg["vocab_size"], H))]
    for label, fn_name, shape in families:
        real = getattr(ops, fn_name)
        if shape is None:
            setattr(ops, fn_name, lambda *a, **k: None)
        else:
            setattr(ops, fn_name, lambda a, w, *r, _real=real, _shape=shape, **k: None if tuple(w.shape) == _shape else _real(a, w, *r, **k))
        try:
            t = timed()
        finally:
            setattr(ops, fn_name, real)
        again = timed()                                  # the whole step once more: clocks drift under a long load
        per_step = ((whole + again) / 2 - t) * 1000
        whole = again
        key = "marginal_us_per_step" if label == "output head" else "marginal_us_per_layer"
        out[key][label] = per_step if label == "output head" else per_step / L
    out["ms_per_step_at_the_end"] = whole
    print(json.dumps(out))
    return 0


def marginal_costs_prefill(args) -> int:
    """Times the step that runs one whole prompt, then the same step with one kernel family's launches left out."""
    import numpy as np
    import torch
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.kernels import ops
    from rustingstrata_b200.sampling import SamplingParams
    cfg = dict(QWEN3_8B)
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    L, S = cfg["num_hidden_layers"], args.prompt_len
    eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=2 * S + 64, max_batch_tokens=S, max_seqs=2)
    eng.lookahead = False
    rng = np.random.default_rng(0)
    prompt = rng.integers(0, cfg["vocab_size"], size=S).tolist()

    def once():
        rid = eng.add_request(prompt, 1, SamplingParams())
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        ev0.record()
        eng.step()
        ev1.record()
        torch.cuda.synchronize()
        eng.drain()
        for r in list(eng.scheduler.running):
            eng.scheduler.running.remove(r)
            eng.runner.release(r.rid)
            eng._samplers.pop(r.rid, None)
        return ev0.elapsed_time(ev1)

    def timed():
        return float(np.median([once() for _ in range(max(5, args.steps // 8))]))
    for _ in range(3):
        timed()
    whole = timed()
    H, I = cfg["hidden_size"], cfg["intermediate_size"]
    qkv = (cfg["num_attention_heads"] + 2 * cfg["num_key_value_heads"]) * cfg["head_dim"]
    out = {"prompt_len": S, "layers": L, "ms_per_step": whole, "us_per_layer": whole / L * 1000, "marginal_us_per_layer": {},
           "marginal_us_per_step": {}}
    families = [("attention of the portion", "attention_prefill", None), ("qk_norm_rope_kv", "qk_norm_rope_kv", None),
                ("gate/up product", "linear_swiglu", None), ("row norms (+ owed sums)", "rmsnorm", None),
                ("qkv product", "linear", (qkv, H)), ("output product", "linear", (H, cfg["num_attention_heads"] * cfg["head_dim"])),
                ("down product", "linear", (H, I)), ("output head", "linear", (cfg["vocab_size"], H))]
    for label, fn_name, shape in families:
        real = getattr(ops, fn_name)
        if shape is None:
            setattr(ops, fn_name, lambda *a, **k: None)
        else:
            setattr(ops, fn_name, lambda a, w, *r, _real=real, _shape=shape, **k: None if tuple(w.shape) == _shape else _real(a, w, *r, **k))
        try:
            t = timed()
        finally:
            setattr(ops, fn_name, real)
        again = timed()
        per_step = ((whole + again) / 2 - t) * 1000
        whole = again
        key = "marginal_us_per_step" if label == "output head" else "marginal_us_per_layer"
        out[key][label] = per_step if label == "output head" else per_step / L
    out["ms_per_step_at_the_end"] = whole
    print(json.dumps(out))
    return 0


def lokinex_config(width: int) -> dict:
    """A Lokinex model whose layers resemble real ones at this width: latent attention with a 4:1 latent (rank width / 4,
    heads of 64 + 64 query/key and 128 value coordinates), recurrent layers 5/4 of the width in blocks of 256, a dense
    feed-forward of 4 x width, 32 experts of 3/4 width with 4 per token and a shared expert of twice that; four layers
    (attention + dense, recurrence + experts, attention + experts, recurrence + experts) run twice by the loop."""
    heads = width // 128
    att = {"type": "latent_attention", "mixer": {"heads": heads, "dim": 64, "rot_dim": 64, "vdim": 128, "kv_rank": width // 4,
                                                 "rot": {"base": 1000000.0, "dims": 64}, "scale": 128 ** -0.5}}
    rec = {"type": "rglru", "mixer": {"width": width * 5 // 4, "blocks": width * 5 // 4 // 256, "conv": 4}}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": width * 3 // 4}, "shared": {"ff": width * 3 // 2}}
    dense = {"kind": "dense", "ff": 4 * width}
    return {"architecture": "Lokinex", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "canon": {"taps": 4},
            "layers": [dict(att, mlp=dense), dict(rec, mlp=moe), dict(att, mlp=moe), dict(rec, mlp=moe)],
            "loop": {"start": 0, "stop": 4, "times": 2}}


TABEDRA_WINDOW = 1024


def tabedra_config(width: int) -> dict:
    """A Tabedra model whose layers resemble real ones at this width: heads of 128 query/key and 128 value coordinates,
    one key/value head per four query heads, convolutions of 4 taps, a sliding window of 1,024 keys with a distance-bias
    table of 32 rows, four residual streams, 32 squared-ReLU experts as wide as the model with 4 per token and a shared
    expert of twice that; eight layers, of which every second pair reads the keys and values of the layer before it."""
    heads = width // 128
    mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "conv": 4, "scale": 0.5,
             "bias_max": float(TABEDRA_WINDOW), "bias_rows": 32, "mask": {"size": TABEDRA_WINDOW}}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": width}, "shared": {"ff": 2 * width}}
    layers = []
    for i in range(8):
        m = dict(mixer)
        if i % 4 >= 2:
            m["kv_from"] = i - i % 4 + 1
        layers.append({"type": "attention", "mixer": m, "mlp": moe})
    return {"architecture": "Tabedra", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "streams": 4,
            "max_positions": 8192, "embedding": {"bigram": {"buckets": 65521, "mul_prev": 31337, "mul_cur": 7919}},
            "layers": layers}


def kupelix_config(width: int) -> dict:
    """A Kupelix model whose layers resemble real ones at this width: heads of 128 query/key and 128 value coordinates
    in all three mixers; attention with one key/value head per four query heads and half of each head rotated; the delta
    rule with one query/key head per two state heads, 4 taps and low-rank maps of 64; a dense feed-forward of 4 x width
    in every layer; four layers (attention, delta rule, HGRN2, attention) run twice by the loop."""
    heads = width // 128
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128,
                                          "scale": 128 ** -0.5, "rot": {"base": 1000000.0, "dims": 64}}}
    delta = {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128,
                                                "conv": 4, "decay_rank": 64, "gate_rank": 64}}
    hgrn = {"type": "hgrn2", "mixer": {"heads": heads, "dim": 128, "vdim": 128}}
    dense = {"kind": "dense", "ff": 4 * width}
    return {"architecture": "Kupelix", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
            "layers": [dict(att, mlp=dense), dict(delta, mlp=dense), dict(hgrn, mlp=dense), dict(att, mlp=dense)],
            "loop": {"start": 0, "stop": 4, "times": 2}}


KOZASUN_MASK = 1024


def kozasun_config(width: int) -> dict:
    """A Kozasun model whose layers resemble real ones at this width: heads of 128 query/key and 128 value coordinates in
    all three mixers; attention with one key/value head per four query heads, half of each head rotated and blocks of
    1,024 positions; retention with decays 1 - 2^-(5 + h); latent attention over a latent of width / 4 with a window of
    1,024 keys; a dense feed-forward of 4 x width or 32 experts of 3/4 width in 4 groups of which 2 are kept, 4 per token,
    and a shared expert of 3/2 width; two residual streams; eight layer runs (attention + dense, retention + experts,
    latent attention + dense, latent attention + experts, twice, the second attention layer with the first one's tensors)."""
    heads = width // 128
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128,
                                          "scale": 128 ** -0.5, "rot": {"base": 1000000.0, "dims": 64}, "mask": {"size": KOZASUN_MASK}}}
    ret = {"type": "retention", "mixer": {"heads": heads, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128},
                                          "decay": [1.0 - 2.0 ** -(5 + h % 8) for h in range(heads)]}}
    lat = {"type": "latent_attention", "mixer": {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": width // 4,
                                                 "scale": 128 ** -0.5, "mask": {"size": KOZASUN_MASK}}}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4, "scale": 2.5, "groups": {"count": 4, "keep": 2}},
           "expert": {"ff": width * 3 // 4}, "shared": {"ff": width * 3 // 2}}
    dense = {"kind": "dense", "ff": 4 * width}
    return {"architecture": "Kozasun", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "streams": 2,
            "embedding": {"scale": 1.0}, "max_positions": 8192,
            "layers": [dict(att, mlp=dense), dict(ret, mlp=moe), dict(lat, mlp=dense), dict(lat, mlp=moe),
                       dict(att, mlp=dense, weights_of=0), dict(ret, mlp=moe), dict(lat, mlp=dense), dict(lat, mlp=moe)]}


SEFELORN_WINDOW = 1024


def sefelorn_config(width: int) -> dict:
    """A Sefelorn model whose layers resemble real ones at this width: attention heads of 128 query/key and 128 value
    coordinates with one key/value head per four query heads, half of each head rotated, a window of 1,024 keys that keeps
    the first 16 tokens, beside gated linear attention with as many heads of 128 + 128 and a low-rank map of 16; Mamba-2
    with twice the width inside, heads of 64, states of 128 rows, one group, 4 taps; a gated feed-forward of 8/3 width (as
    many weights as two matrices of 4 x width); four layers (parallel, Mamba-2, parallel, Mamba-2) run twice by the loop."""
    heads = width // 128
    par = {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "rot": {"base": 1000000.0, "dims": 64}, "mask": {"size": SEFELORN_WINDOW, "keep_first": 16}},
        "right": {"heads": heads, "dim": 128, "vdim": 128, "tau": 16.0, "decay_rank": 16}, "left_scale": 0.5, "right_scale": 0.5}}
    mamba = {"type": "mamba2", "mixer": {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}}
    dense = {"kind": "dense", "ff": width * 8 // 3 // 64 * 64, "limit": 7.0}
    return {"architecture": "Sefelorn", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "logit_scale": 1.0, "layers": [dict(par, mlp=dense), dict(mamba, mlp=dense), dict(par, mlp=dense), dict(mamba, mlp=dense)],
            "loop": {"start": 0, "stop": 4, "times": 2}}


def gemodra_config(width: int) -> dict:
    """A Gemodra model whose layers resemble real ones at this width: latent attention with heads of 128 query/key and 128
    value coordinates over a latent of width / 4, with 64 rotated ones besides and queries through a latent of 3/4 width in
    two layers of three, without positions and queries through half the width in the third; 32 experts of 3/4 width and 8
    identity experts in 4 groups of which 2 are kept, 4 per token, and a shared expert of 3/2 width; a per-layer token input
    of width / 8; eight layers."""
    heads = width // 128
    rot = {"type": "latent_attention", "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": width // 4,
                                                 "q_rank": width * 3 // 4, "scale": 192 ** -0.5, "rot": {"base": 1000000.0, "dims": 64}}}
    flat = {"type": "latent_attention_2", "mixer": {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": width // 4,
                                                    "q_rank": width // 2, "scale": 128 ** -0.5}}
    moe = {"kind": "moe", "router": {"experts": 32, "identity": 8, "top": 4, "scale": 2.5, "groups": {"count": 4, "keep": 2}},
           "expert": {"ff": width * 3 // 4}, "shared": {"ff": width * 3 // 2}}
    return {"architecture": "Gemodra", "vocab": 32768, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
            "token_side": {"dim": width // 8}, "logit_softcap": 30.0, "max_positions": 8192,
            "layers": [dict(flat if i % 3 == 2 else rot, mlp=moe) for i in range(8)]}


def qwen3_windowed(width: int) -> dict:
    """The closest existing model for the Tabedra design: the Qwen3 decoder of :func:`qwen3_like` with the same sliding
    window on every layer and as many key/value heads."""
    heads = width // 128
    return dict(qwen3_like(width), num_key_value_heads=max(1, heads // 4), use_sliding_window=True,
                sliding_window=TABEDRA_WINDOW, max_window_layers=0, layer_types=["sliding_attention"] * 8)


def qwen3_like(width: int) -> dict:
    """The closest existing model at equal size: as many layer runs (8), the same width, vocabulary and head size, a gated
    feed-forward with as many weights as the dense one above (3 matrices of 8/3 width against 2 of 4 width)."""
    return dict(QWEN3_8B, vocab_size=32768, hidden_size=width, num_hidden_layers=8, num_attention_heads=width // 128,
                num_key_value_heads=max(1, width // 512), head_dim=128, intermediate_size=width * 8 // 3 // 64 * 64,
                max_position_embeddings=8192)


class OpTimer:
    """Device time per launcher of ``kernels.ops`` inside a region: CUDA events around every call of the listed
    launchers (eager steps only), summed per name after a synchronisation."""
    NAMES = ("embed", "rmsnorm", "rmsnorm_add", "concat_embed", "short_conv", "block_linear", "gated_linear_recurrence",
             "gated_linear_recurrence_gates", "latent_kv_write", "relu_squared", "moe_route", "grouped_linear", "moe_combine",
             "grouped_gemm_mma", "attention_latent", "linear", "linear_swiglu", "qk_norm_rope_kv", "attention_prefill", "attention_decode",
             "attention_decode_items", "silu_mul", "residual_add", "sample", "latent_expand", "embed_sum", "stream_layernorm",
             "stream_update", "router_topk", "conv_norm_kv_write", "sigmoid_gate", "talking_attention_prep", "talking_attention", "talking_attention_mma", "grouped_attention_mma",
             "state_recurrence", "state_recurrence_chunked", "hgrn2_prep", "delta_prep", "head_norm_gate", "activation", "scale_rows", "retention_prep",
             "mamba2_prep", "low_rank_decay", "pad_heads", "gated_group_norm", "add_embed", "embed_rmsnorm",
             "gelu_table_gate", "cast_rows", "softcap_rows", "router_route", "latent_queries")

    def __init__(self):
        self.events, self.real = [], {}

    def __enter__(self):
        import torch
        from rustingstrata_b200.kernels import ops
        for name in self.NAMES:
            fn = getattr(ops, name, None)
            if fn is None:
                continue
            self.real[name] = fn

            def timed(*a, _fn=fn, _name=name, **k):
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                out = _fn(*a, **k)
                e1.record()
                self.events.append((_name, e0, e1))
                return out
            setattr(ops, name, timed)
        return self

    def __exit__(self, *exc):
        from rustingstrata_b200.kernels import ops
        for name, fn in self.real.items():
            setattr(ops, name, fn)

    def totals(self):
        import torch
        torch.cuda.synchronize()
        out = {}
        for name, e0, e1 in self.events:
            t = out.setdefault(name, [0, 0.0])
            t[0] += 1
            t[1] += e0.elapsed_time(e1) * 1000
        return {k: {"calls": v[0], "us": round(v[1], 1)} for k, v in sorted(out.items(), key=lambda kv: -kv[1][1])}


def lokinex_workload(args, design: str = "lokinex") -> int:
    """Prefill of one 2,048-token prompt and decode at batch 8 (2,048 tokens held each) of the Lokinex (or Tabedra) design
    at layer sizes that resemble a real model's, beside the Qwen3 dense decoder at equal width, depth and vocabulary (for
    Tabedra: with the same sliding window); device time per kernel family of one prompt step and one decode step of each
    (eager steps with events around every launcher)."""
    import numpy as np
    import torch
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.engine import StepEntry, roofline
    from rustingstrata_b200.sampling import SamplingParams
    pk = roofline.peaks(os.path.join(ROOT, "MEASURED_PEAKS.json"))
    clocks = ClockSampler()
    clocks.start()
    pair = {"lokinex": (lokinex_config, qwen3_like), "tabedra": (tabedra_config, qwen3_windowed),
            "kupelix": (kupelix_config, qwen3_like), "kozasun": (kozasun_config, kupelix_config),
            "sefelorn": (sefelorn_config, kupelix_config), "gemodra": (gemodra_config, kozasun_config)}[design]
    out = {"workload": design, "prompt_len": PROMPT, "batch": args.batch, "steps": args.steps, "dtype": "bf16",
           "data": "synthetic", "weights": "random N(0,0.02) bf16", "peaks": pk["source"], "sizes": {}}
    for width in [int(x) for x in args.sizes.split(",")]:
        rec = {}
        # the closest existing model of the design
        other = {"kozasun": "kupelix", "sefelorn": "kupelix", "gemodra": "kozasun"}.get(design, "qwen3")
        for name, cfg in ((design, pair[0](width)), (other, pair[1](width))):
            V = cfg.get("vocab", cfg.get("vocab_size"))
            eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=args.batch * CONTEXT,
                         max_batch_tokens=PROMPT, max_seqs=args.batch)
            runner = eng.runner
            rng = np.random.default_rng(0)

            def finish_all():
                eng.drain()
                for r in list(eng.scheduler.running):
                    eng.scheduler.running.remove(r)
                    runner.release(r.rid)
                    eng._samplers.pop(r.rid, None)

            def prompt_ms():
                eng.add_request(rng.integers(0, V, size=PROMPT).tolist(), CONTEXT - PROMPT, SamplingParams())
                eng.lookahead = False
                ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                ev0.record()
                eng.step()
                ev1.record()
                torch.cuda.synchronize()
                eng.lookahead = True
                finish_all()
                return ev0.elapsed_time(ev1)
            for _ in range(3):
                prompt_ms()
            pms = float(np.median([prompt_ms() for _ in range(5)]))
            flops = roofline.step_flops(runner.model, [PROMPT], [PROMPT], 1)
            for _ in range(args.batch):
                eng.add_request(rng.integers(0, V, size=PROMPT).tolist(), CONTEXT - PROMPT, SamplingParams())
            while eng.scheduler.waiting or any(r.prefilling for r in eng.scheduler.running):
                eng.step()
            for _ in range(args.warmup):
                eng.step()
            kv_tokens = sum(runner.length(r.rid) for r in eng.scheduler.running)
            dms = eng.decode_steps_device_timed(args.steps, warmup=3)
            launches = eng.kernels_in_timed_steps / args.steps
            dec = roofline.decode_roofline(runner.model, runner.kv_bytes_per_token, kv_tokens, dms, pk)
            # device time per launcher: one eager decode step of the same batch, one eager prompt step
            eng.drain()
            graphs, runner.use_graphs = runner.use_graphs, False
            with OpTimer() as t_dec:
                for _ in range(3):
                    eng.step()
                eng.drain()
                t_dec.events.clear()
                eng.step()
                eng.drain()
            dec_ops = t_dec.totals()
            finish_all()
            with OpTimer() as t_pre:
                prompt_ms()
                t_pre.events.clear()
                prompt_ms()
            pre_ops = t_pre.totals()
            runner.use_graphs = graphs
            rec[name] = {
                "prefill_tok_s": PROMPT / pms * 1000, "prefill_ms": pms, "prefill_tflops": flops / pms / 1e9,
                "prefill_frac_of_tensor_peak": flops / (pms / 1000) / (pk["bf16_tflops"] * 1e12),
                "decode_tok_s": args.batch / dms * 1000, "decode_ms_per_step": dms, "decode_launches_per_step": launches,
                "decode_gbs": dec["achieved"], "decode_frac_of_hbm_peak": dec["frac"],
                "weight_mb": roofline.weight_bytes(runner.model) / 1e6, "kv_bytes_per_token": runner.kv_bytes_per_token,
                "prefill_step_us_by_launcher": pre_ops, "decode_step_us_by_launcher": dec_ops}
            del eng, runner
            torch.cuda.empty_cache()
        out["sizes"][str(width)] = rec
    out["clocks"] = clocks.stop()
    print(json.dumps(out))
    return 0


def _flat_config(name, cfg, n_layers, full_layers, **more):
    out = {"model": name, "layers": n_layers, "layers_of_config": full_layers, "hidden": cfg["hidden_size"],
           "q_heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
           "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "page_size": 16,
           "parallelism": "single-gpu", "weights": "random N(0,0.02) bf16"}
    out.update(more)
    return out


def mixed_workload(args) -> int:
    """Qwen3-14B layer sizes: 32 requests, prompts U[128, 4096], portions of 512 beside decode tokens, 256 tokens each
    at temperature 0.7, context 8,192, all through the engine's own scheduler and entry point."""
    import numpy as np
    import torch
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.engine import roofline
    from rustingstrata_b200.sampling import SamplingParams
    cfg = dict(QWEN3_14B)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    n_req, ctx, chunk, n_new = 32, 8192, 512, 256
    pk = roofline.peaks(os.path.join(ROOT, "MEASURED_PEAKS.json"))
    eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=n_req * ctx, max_batch_tokens=chunk + n_req,
                 max_seqs=n_req, prefill_chunk=chunk)
    rng = np.random.default_rng(1)
    V = cfg["vocab_size"]

    def run(seed):
        lens = rng.integers(128, 4097, size=n_req)
        rids = [eng.add_request(rng.integers(0, V, size=int(n)).tolist(), n_new, SamplingParams(temp=0.7, seed=seed + i))
                for i, n in enumerate(lens)]
        first, steps = {}, []
        launch = eng._launch

        def spy(batch, prev):
            steps.append((sum(len(s.tokens) for s in batch if len(s.tokens) > 1 or s.request.prefilling),
                          sum(1 for s in batch if len(s.tokens) == 1 and not s.request.prefilling)))
            return launch(batch, prev)
        eng._launch = spy
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        generated = 0
        while eng.has_work():
            eng.step()
            now = time.perf_counter()
            for r in eng.scheduler.running:
                if r.generated and r.rid not in first:
                    first[r.rid] = now - t0
        torch.cuda.synchronize()
        wall = time.perf_counter() - t0
        eng._launch = launch
        eng.runner.check_status()
        for rid in rids:
            first.setdefault(rid, wall)
        generated = n_req * n_new
        return wall, generated, int(lens.sum()), sorted(first.values()), steps

    run(100)                                   # warm-up: every kernel shape and graph of the workload has run once
    clocks = ClockSampler()
    clocks.start()
    wall, generated, prompt_tokens, ttft, steps = run(200)
    clk = clocks.stop()
    pre = [p for p, d in steps]
    dec = [d for p, d in steps]
    mix = {"steps": len(steps), "steps_with_prompt_tokens": sum(1 for p in pre if p), "steps_decode_only": sum(1 for p in pre if not p),
           "steps_mixed": sum(1 for p, d in steps if p and d), "prompt_tokens_per_step_mean": float(np.mean([p for p in pre if p] or [0])),
           "decode_tokens_per_step_mean": float(np.mean(dec)), "decode_tokens_per_step_max": int(max(dec))}
    rec = {"metric": "total generated tok/s, continuous batch of 32 (Qwen3-14B sizes, bf16, random weights)",
           "value": generated / wall, "unit": "tok/s", "n_gpus": 1, "higher_is_better": True, "dtype": "bf16",
           "data": "synthetic", "workload": "14b-mixed", "wall_s": wall, "generated_tokens": generated,
           "prompt_tokens": prompt_tokens, "all_tokens_per_s": (generated + prompt_tokens) / wall,
           "ttft_s": {"mean": float(np.mean(ttft)), "max": float(ttft[-1]), "min": float(ttft[0])},
           "step_mix": mix, "preemptions": eng.scheduler.preemptions,
           "config": _flat_config("qwen3-14b-sizes", cfg, cfg["num_hidden_layers"], full_layers, requests=n_req, seq_len=ctx,
                                  prompt_len="U[128,4096]", chunk=chunk, new_tokens=n_new, temperature=0.7,
                                  peaks=pk["source"]),
           "clocks": clk}
    print(json.dumps(rec))
    return 0


def long_context_workload(args) -> int:
    """Qwen3-32B layer sizes: 8 requests with 12,000-token prompts, then 256 greedy tokens each, context 16,384."""
    import numpy as np
    import torch
    from rustingstrata_b200 import Engine
    from rustingstrata_b200.engine import roofline
    from rustingstrata_b200.sampling import SamplingParams
    cfg = dict(QWEN3_32B)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    n_req, ctx, prompt, n_new = 8, 16384, 12000, 256
    pk = roofline.peaks(os.path.join(ROOT, "MEASURED_PEAKS.json"))
    eng = Engine(cfg, dtype="bfloat16", random_seed=0, page_size=16, max_tokens=n_req * ctx, max_batch_tokens=2048,
                 max_seqs=n_req)
    runner = eng.runner
    rng = np.random.default_rng(2)
    V = cfg["vocab_size"]

    def prefill(n_tokens):
        for _ in range(n_req):
            eng.add_request(rng.integers(0, V, size=n_tokens).tolist(), ctx - n_tokens, SamplingParams())
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        while eng.scheduler.waiting or any(r.prefilling for r in eng.scheduler.running):
            eng.step()
        torch.cuda.synchronize()
        return time.perf_counter() - t0

    def finish_all():
        eng.drain()
        for r in list(eng.scheduler.running):
            eng.scheduler.running.remove(r)
            runner.release(r.rid)
            eng._samplers.pop(r.rid, None)

    # the same decode step with next to no cache: what is left of the step when attention has nothing to read
    prefill(16)
    short_ms = eng.decode_steps_device_timed(64, warmup=8)
    finish_all()
    clocks = ClockSampler()
    clocks.start()
    prefill_s = prefill(prompt)
    for _ in range(args.warmup):
        eng.step()
    kv0 = sum(runner.length(r.rid) for r in eng.scheduler.running)
    steps = n_new - args.warmup - 8
    ms = eng.decode_steps_device_timed(steps, warmup=3)
    kv1 = sum(runner.length(r.rid) for r in eng.scheduler.running)
    clk = clocks.stop()
    runner.check_status()
    roof = roofline.decode_roofline(runner.model, runner.kv_bytes_per_token, (kv0 + kv1) / 2.0, ms, pk)
    kv_bytes = (kv0 + kv1) / 2.0 * runner.kv_bytes_per_token
    rec = {"metric": "decode tok/s at batch 8 after 12,000-token prompts (Qwen3-32B sizes, bf16, random weights)",
           "value": n_req / ms * 1000, "unit": "tok/s", "n_gpus": 1, "higher_is_better": True, "dtype": "bf16",
           "data": "synthetic", "workload": "32b-long", "steps": steps, "ms_per_step": ms,
           "roofline": {k: roof[k] for k in ("bound", "achieved", "peak", "unit", "frac")},
           "kv_share_of_bytes": kv_bytes / roof["bytes_per_step"],
           "ms_per_step_at_16_keys": short_ms, "long_cache_share_of_step": (ms - short_ms) / ms,
           "long_cache_gbs": kv_bytes / ((ms - short_ms) / 1000) / 1e9 if ms > short_ms else None,
           "prefill": {"tokens": n_req * prompt, "s": prefill_s, "value": n_req * prompt / prefill_s},
           "config": _flat_config("qwen3-32b-sizes", cfg, cfg["num_hidden_layers"], full_layers, global_batch=n_req,
                                  seq_len=ctx, prompt_len=prompt, new_tokens=n_new, peaks=pk["source"]),
           "clocks": clk}
    print(json.dumps(rec))
    return 0


if __name__ == "__main__":
    sys.exit(main())
