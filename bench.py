#!/usr/bin/env python3
"""Decode and prefill throughput of the SmolLM2-135M shape on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]
                    [--shape 135m|360m|1.7b] [--batch B] [--context C] [--layers L] [--skip-points]
                    [--skip-e2e] [--designs s,m [--only-design llama,nafezen,tazadra,sedopel,selovik,setenex,zadurax]]

A step is one decode step of a batch of 8 sequences whose context ends at 4,096
tokens (prompt 2,048 + 2,048 decoded); ``value`` is decoded tokens per second,
timed with CUDA events over K graph launches: the median of five such regions over
the same range of contexts, as NNIS's own benchmarks take the median of five
(crates/nnis-bench/src/lib.rs:362-428).  ``e2e`` is the same through the Python
entry point with every step's tokens coming from and going back to the host, over
256 steps whatever K is.  The line also carries a 2,048-token prefill, the decode
step's HBM roofline, decoding at batch 1 and 64, and ``kernels``: per kernel of one
more decode step, taken outside every timed region with the kernels' own readings of
the GPU's timer, its launches and the microseconds from its last CTA getting past the
wait for the kernel before to its end, summed over the launches.  Weights are random (seeded),
token ids are uniform random: no checkpoint or dataset is read.
"""
from __future__ import annotations

import argparse
import json
import os
import random
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# The shape of SmolLM2-135M; nothing below the configuration knows these numbers.
SMOLLM2_135M = dict(
    architectures=["LlamaForCausalLM"], model_type="llama", vocab_size=49152, hidden_size=576,
    intermediate_size=1536, num_hidden_layers=30, num_attention_heads=9, num_key_value_heads=3,
    max_position_embeddings=8192, rms_norm_eps=1e-5, rope_theta=100000.0, hidden_act="silu",
    tie_word_embeddings=True, attention_bias=False, torch_dtype="bfloat16")
# The two larger shapes of the same family: what differs from the above.
SHAPES = {
    "135m": ("SmolLM2-135M", {}),
    "360m": ("SmolLM2-360M", dict(num_hidden_layers=32, hidden_size=960, intermediate_size=2560,
                                  num_attention_heads=15, num_key_value_heads=5)),
    "1.7b": ("SmolLM2-1.7B", dict(num_hidden_layers=24, hidden_size=2048, intermediate_size=8192,
                                  num_attention_heads=32, num_key_value_heads=32, rope_theta=130000.0)),
}
CONTEXT = 4096
PROMPT = 2048
BATCH = 8
REPEATS = 5     # timed regions per point; the median is reported
E2E_STEPS = 256  # decode steps of the end-to-end run
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0,
                  "source": "fallback"}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            raw = json.load(f)
        return {"hbm_gbs": float(raw["hbm_gbs"]), "bf16_tflops": float(raw["bf16_tflops"]),
                "bf16_tflops_sustained": float(raw.get("bf16_tflops_sustained", raw["bf16_tflops"])),
                "source": "measured"}
    except (OSError, KeyError, ValueError, TypeError):
        return dict(FALLBACK_PEAKS)


class ClockSampler:
    """nvidia-smi clocks and throttle reasons while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_id: str = "0"):
        """``gpu_id``: what ``nvidia-smi -i`` takes for the GPU that the run is on (its
        UUID: index 0 of this process need not be index 0 of the machine)."""
        self.samples, self.proc, self.gpu_id = [], None, gpu_id

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", self.gpu_id, f"--query-gpu={self.QUERY}",
                 "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), [x.strip() for x in line.split(",")]))

    def mark(self):
        return time.time()

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()

    def summary(self, windows):
        rows = [s for t, s in self.samples if any(a <= t <= b for a, b in windows)] or \
               [s for _, s in self.samples]
        sm = sorted(int(r[0]) for r in rows if r[0].isdigit())
        mx = [int(r[1]) for r in rows if len(r) > 1 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 2 + i and r[2 + i] == "Active"
                                                         for r in rows)]
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(rows), "gpu": self.gpu_id}


def gpu_identity(torch) -> str:
    """The UUID of this process's device 0 in nvidia-smi's spelling; "0" if it cannot be had."""
    try:
        uuid = str(torch.cuda.get_device_properties(0).uuid)
        return uuid if uuid.startswith("GPU-") else "GPU-" + uuid
    except Exception:
        return "0"


def median(values):
    values = sorted(values)
    return values[len(values) // 2]


def write_timeline(path, title, names, rows, marks):
    """The table of one traced step: per launch its begin, first and last CTA past the wait
    for the kernel before, two inner marks, end and duration, relative to the step's first
    begin; then sums per kernel."""
    t0 = min(r[0] for r in rows)
    by_name = {}
    big = 1 << 62
    with open(path, "w") as f:
        f.write(f"# {title}; ns after the step's first CTA\n# launch kernel begin past_wait_first past_wait_last "
                f"mark1_first mark1_last mark2_first mark2_last end duration\n# marks: {marks}\n")
        for i, (name, r) in enumerate(zip(names, rows)):
            rel = [(v - t0 if 0 < v < big else -1) for v in r]
            b, e, w1 = rel[0], rel[1], rel[3]
            f.write(f"{i} {name.replace(' ', '_')} {b} {rel[2]} {w1} {rel[4]} {rel[5]} {rel[6]} {rel[7]} {e} {e - b}\n")
            total = by_name.setdefault(name, [0, 0, 0])
            total[0] += 1
            total[1] += e - b
            total[2] += e - (w1 if w1 >= 0 else b)
        f.write(f"# step: {max(r[1] for r in rows) - t0} ns\n")
        for name, (count, dur, after) in sorted(by_name.items()):
            f.write(f"# {name}: {count} launches, mean begin-to-end {dur / count:.0f} ns, "
                    f"mean last-wait-to-end {after / count:.0f} ns, sum of the latter {after / 1000:.0f} us\n")
    print(open(path).read()[-1800:])


def kernel_times(names, rows):
    """Per kernel of one traced step: launches, and microseconds from the moment its last
    CTA got past the wait for the kernel before to its end (its link in the step's chain),
    summed over the launches; and the step from its first CTA to its last."""
    big = 1 << 62
    out = {}
    for name, r in zip(names, rows):
        begin, end, last_wait = r[0], r[1], r[3]
        start = last_wait if 0 < last_wait < big else begin
        entry = out.setdefault(name, {"launches": 0, "us": 0.0})
        entry["launches"] += 1
        entry["us"] += (end - start) / 1000.0
    for entry in out.values():
        entry["us"] = round(entry["us"], 1)
    out["step"] = {"launches": len(rows), "us": round((max(r[1] for r in rows) - min(r[0] for r in rows)) / 1000.0, 1)}
    return out


def prefill_timeline(engine, path, rng, vocab):
    """One prompt step of 2,048 tokens as the GPU's own timer saw it (the instrumented
    kernels: tcgen05 products, prompt attention, the norms of many rows)."""
    import torch

    from nnis_b200.csrc import ops
    from nnis_b200.engine import SequenceStep
    prompt = [rng.randrange(vocab) for _ in range(PROMPT)]

    def once():
        slot = engine.acquire_slot()
        engine.step([SequenceStep(slot, prompt, [PROMPT - 1])])
        engine.release_slot(slot)
    once()                      # seen once
    buf = ops.trace_begin(4096)
    once()                      # run into its own buffers and captured: both take slots
    names = ops.trace_end()
    for _ in range(3):
        once()
    torch.cuda.synchronize()
    ops.trace_clear()
    once()
    torch.cuda.synchronize()
    half = len(names) // 2
    write_timeline(path, f"one prompt step of {PROMPT} tokens", names[half:], buf[half:2 * half].cpu().tolist(),
                   "products: first operands arrived / all products complete")


def timeline(engine, batch, path, rng, vocab):
    """One decode step at context 4,096 as the GPU's own timer saw it: per launch of the
    decode kernels its begin and end, and when its first and last CTA got past the wait
    for the kernel before, relative to the step's first begin; then sums per kernel."""
    import torch

    from nnis_b200.csrc import ops
    from nnis_b200.engine import SequenceStep
    from nnis_b200.engine.decode import GraphDecoder
    begin = CONTEXT - 16
    slots = [engine.acquire_slot() for _ in range(batch)]
    fed = 0
    while fed < begin:
        n = min(PROMPT, begin - fed)
        per_step = max(1, 16384 // n)
        for i in range(0, batch, per_step):
            engine.step([SequenceStep(s, [rng.randrange(vocab) for _ in range(n)], [])
                         for s in slots[i:i + per_step]])
        fed += n
    dec = GraphDecoder(engine, batch, CONTEXT)
    engine.cache.reserve(slots, [CONTEXT] * batch)
    for r, s in enumerate(slots):
        dec.set_row(r, s, rng.randrange(vocab), begin)
    buf = ops.trace_begin(4096)
    dec.capture()  # the warm-up run takes slots as well; the captured launches take the later half
    names = ops.trace_end()
    for _ in range(4):
        dec.launch()
    torch.cuda.synchronize()
    ops.trace_clear()
    dec.launch()
    torch.cuda.synchronize()
    half = len(names) // 2
    write_timeline(path, f"one decode step, batch {batch}, context {CONTEXT}, {len(dec.chains)} chain(s)",
                   names[half:], buf[half:2 * half].cpu().tolist(),
                   "projections x staged / products done; attention pages done / ticket taken")


# ---------------------------------------------------------------------------
# --designs: the Nafezen, Tazadra, Sedopel, Selovik, Setenex and Zadurax designs beside the Llama decoder at equal width and depth
# ---------------------------------------------------------------------------
def design_configs(size: str):
    """(Llama, Nafezen, Tazadra, Sedopel, Selovik, Setenex, Zadurax) configurations of one width, depth, vocabulary and dense
    feed-forward size; the Nafezen layers alternate latent attention with dense and expert
    feed-forwards and hold one retention layer in four; the Tazadra layers are attention with a
    sink + dense, WKV + experts, selective scan + experts, and attention that reads the first
    layer's keys + dense, twice; the Sedopel layers alternate a pair of mixers (gated softmax
    attention beside lightning attention) + dense with the gated delta rule, which has a dense
    feed-forward every other time; the Selovik layers are differential attention (two maps of half a
    head's size over values of a head's size, a window of 1,024) with dense and expert feed-forwards
    in turn, six layers of which the second and third run twice (eight layer runs); the Setenex layers
    alternate attention with a bias per distance (a window of 1,024 that keeps 64 first tokens) and latent
    attention with queries straight from the input and a window of 1,024, all with experts, six layers
    of which the second and third run twice; the Zadurax layers are a matrix memory, latent attention with a
    sink twice, and attention whose values are its keys (a window of 1,024), all with dense feed-forwards,
    six layers of which the third and fourth run again with a cache of their own."""
    width, heads, ff, layers, q_rank, kv_rank, experts, top = {
        "s": (1024, 16, 2816, 8, 384, 256, 16, 2),
        "m": (2048, 16, 5632, 8, 768, 512, 32, 4),
    }[size]
    dim = width // heads
    llama = dict(architectures=["LlamaForCausalLM"], model_type="llama", vocab_size=32768, hidden_size=width,
                 intermediate_size=ff, num_hidden_layers=layers, num_attention_heads=heads,
                 num_key_value_heads=heads // 4, max_position_embeddings=8192, rms_norm_eps=1e-5,
                 rope_theta=100000.0, hidden_act="silu", tie_word_embeddings=True, attention_bias=False,
                 torch_dtype="bfloat16")
    latent = {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "q_rank": q_rank, "kv_rank": kv_rank,
              "rot": {"base": 10000.0, "dims": dim // 2}, "scale": (dim + dim // 2) ** -0.5}
    ret_heads = max(1, width // 256)
    retention = {"heads": ret_heads, "dim": 128, "vdim": 256, "rot": {"base": 10000.0, "dims": 128},
                 "decay": [1.0 - 2.0 ** (-5 - i % 4) for i in range(ret_heads)]}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff // (2 * top)},
           "shared": {"ff": ff // 2}}
    pattern = [("latent_attention", latent, dense), ("latent_attention", latent, moe),
               ("retention", retention, moe), ("latent_attention", latent, dense)]
    nafezen = {"architecture": "Nafezen", "vocab": 32768, "width": width, "norm": {"eps": 1e-5, "groups": 4},
               "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in (pattern[i % 4] for i in range(layers))]}
    attention = {"heads": heads, "kv_heads": heads // 4, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
                 "softcap": 50.0, "mask": {"size": 1024},
                 "rot": {"base": 500000.0, "dims": dim,
                         "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    wkv = {"heads": width // 64, "dim": 64, "decay_rank": 64}
    scan = {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}
    t_dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    t_moe = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff // (2 * top)}}
    t_layers = []
    for i in range(layers):
        kind, mixer, mlp = [("attention", attention, t_dense), ("wkv", wkv, t_moe), ("mamba1", scan, t_moe),
                            ("attention", {**attention, "kv_from": i - 3}, t_dense)][i % 4]
        t_layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    tazadra = {"architecture": "Tazadra", "vocab": 32768, "width": width, "norm": {"eps": 1e-5},
               "residual_mult": 0.7, "logit_softcap": 40.0, "layers": t_layers}
    softmax = {"heads": heads, "kv_heads": heads // 4, "dim": dim, "vdim": dim, "scale": 4.0 / dim,
               "rot": {"base": 500000.0, "dims": dim // 2}}
    lightning = {"heads": width // 128, "dim": 64, "vdim": 128,
                 "decay": [1.0 - 2.0 ** (-4 - i % 5) for i in range(width // 128)]}
    delta = {"heads": width // 64, "kv_heads": width // 128, "dim": dim, "vdim": 128, "conv": 4}
    s_layers = []
    for i in range(layers):
        kind, mixer, mlp = [("parallel", {"left": softmax, "right": lightning}, dense), ("delta", delta, dense),
                            ("parallel", {"left": softmax, "right": lightning}, dense), ("delta", delta, None)][i % 4]
        s_layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    sedopel = {"architecture": "Sedopel", "vocab": 32768, "width": width, "norm": {"eps": 1e-6}, "layers": s_layers}
    two_maps = {"heads": heads, "kv_heads": heads // 4, "dim": dim // 2, "vdim": dim, "scale": (dim // 2) ** -0.5,
                "diff": 0.8, "mask": {"size": 1024},
                "rot": {"base": 500000.0, "dims": dim // 2,
                        "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    v_moe = {"kind": "moe", "expert": {"ff": ff // (2 * top)}, "shared": {"ff": ff // 2},
             "router": {"experts": experts, "top": top, "identity": experts // 4,
                        "groups": {"count": 4, "keep": 2}}}
    v_layers = [{"type": "attention", "mixer": two_maps, "mlp": dense if i % 2 == 0 else v_moe}
                for i in range(layers - 2)]
    selovik = {"architecture": "Selovik", "vocab": 32768, "width": width, "norm": {"eps": 1e-5},
               "embedding": {"scale": 1.0, "bigram": {"buckets": 8191, "mul_prev": 31, "mul_cur": 17}},
               "logit_scale": 1.0, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": v_layers}
    biased = {"heads": heads, "kv_heads": heads // 4, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "bias_max": 1024,
              "mask": {"size": 1024, "keep_first": 64}}
    direct = {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "kv_rank": kv_rank,
              "rot": {"base": 10000.0, "dims": dim // 2}, "scale": (dim + dim // 2) ** -0.5, "mask": {"size": 1024}}
    x_moe = {"kind": "moe", "expert": {"ff": ff // (2 * top)},
             "router": {"experts": experts, "top": top, "groups": {"count": 4, "keep": 2}}}
    x_layers = [{"type": "attention" if i % 2 == 0 else "latent_attention", "mixer": biased if i % 2 == 0 else direct,
                 "mlp": x_moe} for i in range(layers - 2)]
    setenex = {"architecture": "Setenex", "vocab": 32768, "width": width, "norm": {"eps": 1e-5},
               "embedding": {"scale": 1.0}, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": x_layers}
    memory = {"heads": ret_heads, "dim": 128, "vdim": 256, "gate_cap": 15.0}
    sunk = {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "kv_rank": kv_rank,
            "rot": {"base": 10000.0, "dims": dim // 2,
                    "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
            "scale": (dim + dim // 2) ** -0.5}
    keyed = {"heads": heads, "kv_heads": heads // 4, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
             "mask": {"size": 1024}, "rot": {"base": 10000.0, "dims": dim // 2}}
    pattern = [("mlstm", memory), ("latent_attention", sunk), ("latent_attention", sunk), ("attention", keyed)]
    z_layers = [{"type": pattern[i % 4][0], "mixer": pattern[i % 4][1], "mlp": dense} for i in range(layers)]
    for i in range(layers - 2, layers):
        z_layers[i]["weights_of"] = i - 4
    zadurax = {"architecture": "Zadurax", "vocab": 32768, "width": width, "norm": {"eps": 1e-6}, "layers": z_layers}
    return llama, nafezen, tazadra, sedopel, selovik, setenex, zadurax


DESIGN_NAMES = ("llama", "nafezen", "tazadra", "sedopel", "selovik", "setenex", "zadurax")


def profile_steps(args) -> int:
    """For a profiler (``--designs s --profile-steps N``): N prompt steps of 2,048 tokens and N
    decode steps of 8 sequences at context 2,000 of the first four Nafezen layers, run eagerly
    (no CUDA graph) so that every launch is there to be captured; nothing is timed."""
    import torch

    import nnis_b200.engine.engine as engine_module
    from nnis_b200.engine import Engine, SequenceStep
    from nnis_b200.weights import write_random_model
    engine_module.GRAPH_MIN_TOKENS = 1 << 30
    cfg = design_configs(args.designs.split(",")[0])[DESIGN_NAMES.index(args.profile_design)]
    cfg["layers"] = cfg["layers"][:4]
    rng = random.Random(0)
    with tempfile.TemporaryDirectory() as tmp:
        write_random_model(cfg, seed=0, out_dir=tmp, std=1.0, norm_std=0.1, std_by_fan_in=True)
        engine = Engine.from_dir(tmp, dtype="bfloat16", max_tokens=8 * 2200 + 4096)
    prompt = [rng.randrange(cfg["vocab"]) for _ in range(2048)]
    for _ in range(args.profile_steps):
        slot = engine.acquire_slot()
        engine.step([SequenceStep(slot, prompt, [2047])])
        engine.release_slot(slot)
    slots = [engine.acquire_slot() for _ in range(8)]
    engine.step([SequenceStep(s, prompt[:2000], []) for s in slots])
    for _ in range(args.profile_steps):
        engine.step([SequenceStep(s, [5], [0]) for s in slots])
    torch.cuda.synchronize()
    print(json.dumps({"profile_steps": args.profile_steps, "layers": 4, "design": args.profile_design}))
    return 0


def compare_designs(args) -> int:
    """Prefill and decode of both designs at each size, with the time of every part of a
    prompt step (CUDA events around the part, one eager step) against the part's own
    count of operations; one JSON line per design and size."""
    import torch

    from nnis_b200 import LLM
    from nnis_b200.engine import SequenceStep
    from nnis_b200.engine.decode import GraphDecoder
    from nnis_b200.weights import write_random_model
    pk = peaks()
    rng = random.Random(0)
    prompt_len, context, batch = 2048, 2048, 8
    clocks = ClockSampler(gpu_identity(torch))
    clocks.start()
    windows = []

    def timed(fn, n):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        t0 = clocks.mark()
        start.record()
        for _ in range(n):
            fn()
        end.record()
        torch.cuda.synchronize()
        windows.append((t0, clocks.mark()))
        return start.elapsed_time(end) / n

    for size in args.designs.split(","):
        for name, cfg in zip(DESIGN_NAMES, design_configs(size)):
            if args.only_design and name not in args.only_design.split(","):
                continue
            with tempfile.TemporaryDirectory() as tmp:
                write_random_model(cfg, seed=0, out_dir=tmp, std=1.0, norm_std=0.1, std_by_fan_in=True)
                llm = LLM(tmp, dtype="bfloat16", device_ordinal=0, max_tokens=batch * (context + 64) + 4 * prompt_len,
                          max_batch=batch, pipeline_decode=False)
            engine = llm.engine
            vocab = engine.spec.vocab_size
            prompt = [rng.randrange(vocab) for _ in range(prompt_len)]
            del windows[:]

            def prefill_once():
                slot = engine.acquire_slot()
                engine.step([SequenceStep(slot, prompt, [prompt_len - 1])])
                engine.release_slot(slot)
            for _ in range(3):
                prefill_once()
            prefill_ms = median([timed(prefill_once, 4) for _ in range(REPEATS)])
            flops = engine.model.step_flops([prompt_len], [0], 1)
            # every part of one eager prompt step between events of its own
            parts, marks = {}, []
            saved = []
            for block in engine.model.blocks:
                # (the members of a pair of mixers are timed too, inside the pair's own time)
                for part in [q for p in block.parts() for q in (p, *getattr(p, "members", ()))]:
                    kind = type(part).__name__
                    saved.append((part, part.forward))

                    def wrapped(*a, _f=part.forward, _k=kind, _p=part, **kw):
                        b, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                        b.record()
                        out = _f(*a, **kw)
                        e.record()
                        marks.append((_k, _p, b, e))
                        return out
                    part.forward = wrapped
            import nnis_b200.engine.engine as engine_module
            floor = engine_module.GRAPH_MIN_TOKENS
            engine_module.GRAPH_MIN_TOKENS = 1 << 30  # eager: the events must be in the stream
            try:
                for rep in range(3):
                    marks.clear()
                    prefill_once()
                torch.cuda.synchronize()
            finally:
                engine_module.GRAPH_MIN_TOKENS = floor
                for part, fwd in saved:
                    part.forward = fwd
            for kind, part, b, e in marks:
                entry = parts.setdefault(kind, {"ms": 0.0, "flops": 0.0, "calls": 0})
                entry["ms"] += b.elapsed_time(e)
                entry["flops"] += part.step_flops([prompt_len], [0])
                entry["calls"] += 1
            for entry in parts.values():
                entry["frac_of_bf16_peak"] = round(entry["flops"] / (entry["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4) \
                    if entry["ms"] > 0 else None
                entry["ms"] = round(entry["ms"], 3)
            # decoding: batch 8, contexts ending at 2,048, one CUDA graph a step
            steps, warm = 64, 8
            begin = context - steps - warm
            slots = [engine.acquire_slot() for _ in range(batch)]
            for s in slots:
                engine.step([SequenceStep(s, [rng.randrange(vocab) for _ in range(begin)], [])])
            dec = GraphDecoder(engine, batch, context)
            engine.cache.reserve(slots, [context] * batch)
            regions = []
            snaps = [engine.snapshot(s) for s in slots]
            for rep in range(REPEATS):
                for r, s in enumerate(slots):
                    dec.set_row(r, s, rng.randrange(vocab), begin)
                dec.capture()
                for _ in range(warm):
                    dec.launch()
                regions.append(timed(dec.launch, steps))
            step_ms = median(regions)
            # weights: what one token reads, plus the further experts that a batch's tokens choose
            weight_bytes = engine.model.parameter_bytes()
            for entry in engine.spec.schedule:
                for part in engine.model.blocks[entry.layer].parts():
                    if hasattr(part, "step_bytes"):
                        weight_bytes += part.step_bytes(batch) - part.parameter_bytes()
            step_bytes = weight_bytes + batch * engine.cache.kv_bytes_read(context - steps // 2)
            for s in slots:
                engine.release_slot(s)
            print(json.dumps({
                "design": name, "size": size, "width": engine.spec.hidden_size, "layers": len(engine.spec.layers),
                "layer_runs": len(engine.spec.schedule),
                "weights_read_per_token_mb": round(engine.model.parameter_bytes() / 1e6, 1),
                "weights_read_per_decode_step_mb": round(weight_bytes / 1e6, 1),
                "prefill": {"tokens": prompt_len, "ms": round(prefill_ms, 3), "tok_s": round(prompt_len / (prefill_ms * 1e-3)),
                            "frac_of_bf16_peak": round(flops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
                "prefill_parts": parts,
                "decode": {"batch": batch, "context": context, "ms_per_step": round(step_ms, 4),
                           "tok_s": round(batch / (step_ms * 1e-3)), "launches_per_step": dec.launches_per_step,
                           "frac_of_hbm": round(step_bytes / (step_ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                "clocks": clocks.summary(windows),
                "peaks": pk["source"], "dtype": "bf16", "data": "synthetic (seeded random weights and token ids)"}))
            del llm, engine, dec
            torch.cuda.empty_cache()
    clocks.stop()
    return 0


def main() -> int:
    global CONTEXT
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the shape has")
    ap.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64")
    ap.add_argument("--skip-e2e", action="store_true", help="leave out the end-to-end run")
    ap.add_argument("--batch", type=int, default=BATCH, help="sequences of the main decode point")
    ap.add_argument("--context", type=int, default=CONTEXT,
                    help="tokens at which the decoded contexts end (the metric's: 4096)")
    ap.add_argument("--timeline", metavar="FILE", default=None,
                    help="instead of the benchmark: write the timeline of one decode step of the main "
                         "point (begin, end and wait of every launch of the decode kernels) to FILE; "
                         "with --batch 0, of the 2,048-token prompt step")
    ap.add_argument("--shape", default="135m", choices=sorted(SHAPES),
                    help="layer sizes: the SmolLM2-135M shape (the benchmark) or a larger one of the family")
    ap.add_argument("--designs", metavar="SIZES", default=None,
                    help="instead of the benchmark: the Nafezen, Tazadra, Sedopel, Selovik, Setenex and Zadurax designs beside the Llama decoder at "
                         "equal width and depth, sizes 's' and/or 'm' with commas: prefill, its parts, decoding")
    ap.add_argument("--only-design", metavar="NAMES", default=None,
                    help="with --designs: only these of llama, nafezen, tazadra, sedopel, selovik, setenex, zadurax (commas between them)")
    ap.add_argument("--profile-steps", type=int, default=0,
                    help="with --designs: run this many eager prompt and decode steps of one design's first "
                         "four layers for a profiler instead of the timed comparison")
    ap.add_argument("--profile-design", choices=list(DESIGN_NAMES), default="nafezen",
                    help="with --profile-steps: which design")
    args = ap.parse_args()
    if args.designs:
        return profile_steps(args) if args.profile_steps > 0 else compare_designs(args)
    CONTEXT = max(args.context, 64)
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "Memorithm/NNIS is a Rust workspace (cargo, NVRTC); pip cannot install it "
                          "and no Rust toolchain is present"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch

    from nnis_b200 import LLM
    from nnis_b200.csrc import ops
    from nnis_b200.engine import SequenceStep
    from nnis_b200.engine.decode import GraphDecoder
    from nnis_b200.weights import write_random_model

    pk = peaks()
    cfg = dict(SMOLLM2_135M)
    shape_name, shape_sizes = SHAPES[args.shape]
    cfg.update(shape_sizes)
    cfg["max_position_embeddings"] = max(cfg["max_position_embeddings"], CONTEXT)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    rng = random.Random(0)
    vocab = cfg["vocab_size"]
    K, W = args.steps, args.warmup
    clocks = ClockSampler(gpu_identity(torch))
    windows = []

    with tempfile.TemporaryDirectory() as tmp:
        write_random_model(cfg, seed=0, out_dir=tmp, std=1.0, norm_std=0.1, std_by_fan_in=True)
        most_rows = max(args.batch, 1, 1 if args.skip_points or args.timeline else 64)  # the cache holds the largest point
        llm = LLM(tmp, dtype="bfloat16", device_ordinal=0, max_tokens=max(most_rows * (CONTEXT + 64), 4 * (PROMPT + 64)),
                  max_batch=max(most_rows, 1), pipeline_decode=False)
        engine = llm.engine
        spec = engine.spec
        kv_bytes_per_token = engine.cache.kv_bytes_per_token()
        weight_bytes = engine.model.parameter_bytes()
        clocks.start()

        def timed(fn, n):
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            t0 = clocks.mark()
            start.record()
            for _ in range(n):
                fn()
            end.record()
            torch.cuda.synchronize()
            windows.append((t0, clocks.mark()))
            return start.elapsed_time(end)

        def decode_point(batch, steps, warmup, traced=False):
            """Device-timed decode: the contexts end at CONTEXT after the timed steps.
            ``traced``: afterwards one more step with the kernels' own clock readings
            (outside every timed region), summed per kernel."""
            begin = CONTEXT - steps - warmup
            slots = [engine.acquire_slot() for _ in range(batch)]
            fed = 0
            while fed < begin:  # fill the cache in chunks of at most 2,048 tokens per sequence
                n = min(PROMPT, begin - fed)
                per_step = max(1, 16384 // n)
                for i in range(0, batch, per_step):
                    engine.step([SequenceStep(s, [rng.randrange(vocab) for _ in range(n)], [])
                                 for s in slots[i:i + per_step]])
                fed += n
            dec = GraphDecoder(engine, batch, CONTEXT)
            engine.cache.reserve(slots, [CONTEXT] * batch)
            regions = []
            for rep in range(REPEATS):  # every region decodes the same positions again
                for r, s in enumerate(slots):
                    dec.set_row(r, s, rng.randrange(vocab), begin)
                dec.capture()
                for _ in range(warmup):
                    dec.launch()
                before = ops.launch_count()
                regions.append(timed(dec.launch, steps))
                launches = dec.launches_per_step * steps + (ops.launch_count() - before)
            ms = median(regions)
            kernels = None
            if traced:
                seen = GraphDecoder(engine, batch, CONTEXT)  # (its launches get slots of the trace at capture)
                for r, s in enumerate(slots):
                    seen.set_row(r, s, rng.randrange(vocab), begin)
                buf = ops.trace_begin(4096)
                seen.capture()  # the warm-up run takes slots as well; the captured launches the later half
                names = ops.trace_end()
                for _ in range(3):
                    seen.launch()
                torch.cuda.synchronize()
                ops.trace_clear()
                seen.launch()
                torch.cuda.synchronize()
                half = len(names) // 2
                kernels = kernel_times(names[half:], buf[half:2 * half].cpu().tolist())
            for s in slots:
                engine.release_slot(s)
            mean_context = CONTEXT - (steps + 1) / 2.0
            step_bytes = weight_bytes + batch * mean_context * kv_bytes_per_token
            return {"tok_s": batch * steps / (ms * 1e-3), "ms_per_step": ms / steps,
                    "launches": launches, "bytes_per_step": step_bytes,
                    "gbs": step_bytes / (ms / steps * 1e-3) / 1e9,
                    "spread": (max(regions) - min(regions)) / ms, "kernels": kernels}

        if args.timeline:
            if args.batch == 0:
                prefill_timeline(engine, args.timeline, rng, vocab)
            else:
                timeline(engine, args.batch, args.timeline, rng, vocab)
            clocks.stop()
            return 0
        main_point = decode_point(args.batch, K, W, traced=True)

        # -- prefill of 2,048 tokens ------------------------------------------------
        prompt = [rng.randrange(vocab) for _ in range(PROMPT)]

        def prefill_once():
            slot = engine.acquire_slot()
            engine.step([SequenceStep(slot, prompt, [PROMPT - 1])])
            engine.release_slot(slot)

        for _ in range(3):
            prefill_once()
        # regions of four prompts one after another: the host's preparation of the next
        # step runs under the GPU's work on this one, as in a server that has prompts waiting
        prefill_ms = median([timed(prefill_once, 4) for _ in range(REPEATS)]) / 4
        prefill_flops = engine.model.step_flops([PROMPT], [0], 1)  # what the parts say they compute
        prefill_rate = prefill_flops / (prefill_ms * 1e-3)
        prefill = {"value": PROMPT / (prefill_ms * 1e-3), "tokens": PROMPT, "ms": prefill_ms,
                   "frac": prefill_rate / (pk["bf16_tflops"] * 1e12),
                   "frac_of_sustained": prefill_rate / (pk["bf16_tflops_sustained"] * 1e12),
                   "tflops": prefill_rate / 1e12}

        # -- end to end: host tokens in and out every step -----------------------------
        e2e = None
        if not args.skip_e2e:
            e2e_new = E2E_STEPS + 1
            prompts = [[rng.randrange(vocab) for _ in range(CONTEXT - e2e_new)] for _ in range(args.batch)]
            llm.generate([p[:64] for p in prompts], max_new_tokens=4, stop_token_ids=())
            llm.backend._decoder(args.batch, CONTEXT, False).capture()  # the graph the timed run will launch
            stamps = []
            h2d0, d2h0 = llm.backend.h2d_bytes + engine.h2d_bytes, llm.backend.d2h_bytes
            first_done = {}

            def on_token(i, t):
                if i not in first_done:
                    first_done[i] = True
                    if len(first_done) == args.batch:
                        torch.cuda.synchronize()
                        stamps.append((time.perf_counter(), llm.backend.h2d_bytes + engine.h2d_bytes,
                                       llm.backend.d2h_bytes))
            t0 = clocks.mark()
            results = llm.generate(prompts, max_new_tokens=e2e_new, stop_token_ids=(), on_token=on_token)
            torch.cuda.synchronize()
            t_end = time.perf_counter()
            windows.append((t0, clocks.mark()))
            assert all(r.ok and len(r.token_ids) == e2e_new for r in results), \
                [r.error for r in results if not r.ok]
            t_first, h2d1, d2h1 = stamps[0]
            e2e_steps = e2e_new - 1
            e2e = {"value": args.batch * e2e_steps / (t_end - t_first), "unit": "tokens/s",
                   "h2d_bytes_per_step": (llm.backend.h2d_bytes + engine.h2d_bytes - h2d1) // e2e_steps,
                   "d2h_bytes_per_step": (llm.backend.d2h_bytes - d2h1) // e2e_steps,
                   "steps": e2e_steps}

        points = {}
        if not args.skip_points:
            p1 = decode_point(1, min(K, 256), W)
            p64 = decode_point(64, min(K, 64), W)
            points = {"decode_b1": p1["tok_s"], "decode_b64": p64["tok_s"],
                      "decode_b1_hbm_frac": p1["gbs"] / pk["hbm_gbs"],
                      "decode_b64_hbm_frac": p64["gbs"] / pk["hbm_gbs"]}
            # the regime of the reference's own published runs: one 3-token prompt, 32
            # greedy tokens, wall clock around generate() (median of 5 after 2 warm-ups)
            short = [rng.randrange(vocab) for _ in range(3)]
            walls = []
            for i in range(7):
                torch.cuda.synchronize()
                t_a = time.perf_counter()
                out = llm.generate([short], max_new_tokens=32, stop_token_ids=())
                torch.cuda.synchronize()
                if i >= 2:
                    walls.append(time.perf_counter() - t_a)
                assert out[0].ok and len(out[0].token_ids) == 32
            points["generate_3_plus_32_ms"] = sorted(walls)[len(walls) // 2] * 1e3
            points["generate_3_plus_32_tok_s"] = 32 / sorted(walls)[len(walls) // 2]
        clocks.stop()

    line = {
        "metric": f"decode tok/s @ batch {args.batch}, context {CONTEXT} ({shape_name} bf16)",
        "value": main_point["tok_s"], "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W,
        "ms_per_step": main_point["ms_per_step"], "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (seeded random weights and token ids)",
        "impl": "ours",
        "config": {"model": f"{shape_name} shape", "global_batch": args.batch, "seq_len": CONTEXT,
                   "parallelism": "single GPU", "prompt_len": PROMPT, "layers": cfg["num_hidden_layers"],
                   "layers_of_shape": full_layers, "hidden_size": cfg["hidden_size"],
                   "intermediate_size": cfg["intermediate_size"], "heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg.get("head_dim") or cfg["hidden_size"] // cfg["num_attention_heads"],
                   "vocab_size": vocab, "rope_theta": cfg["rope_theta"],
                   "rms_norm_eps": cfg["rms_norm_eps"], "tied_embeddings": True,
                   "cache_page_tokens": 64, "l2": "inputs larger than L2 (weights + KV per step)",
                   "peaks": pk["source"], "timing": f"median of {REPEATS} regions of K steps"},
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": main_point["gbs"], "peak": pk["hbm_gbs"],
                     "unit": "GB/s", "frac": main_point["gbs"] / pk["hbm_gbs"]},
        "points": points,
        "spread": main_point["spread"],
        "e2e": e2e,
        "gpu_launches": main_point["launches"],
        "kernels": main_point["kernels"],
        "clocks": clocks.summary(windows),
    }
    try:  # where the numbers were taken (NNIS's benchmarks carry such a record too)
        line["environment"] = {"gpu": torch.cuda.get_device_name(0), "cuda": torch.version.cuda,
                               "torch": torch.__version__, "python": sys.version.split()[0]}
    except Exception:  # the record is a courtesy; the measurement stands without it
        pass
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
