#!/usr/bin/env python3
"""Headline measurement: GPT-2 124M, random weights, one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--dtype bf16|fp32] [--impl reference]

A "step" is one decode step of a batch of 8 sequences near the model's full context.  The
line printed is one JSON object: ``value`` = decoded tokens per second on the device (CUDA
events around exactly K captured steps), ``e2e`` = the same through the Python entry point
``Engine.generate`` with host tokens in and out, plus

* ``prefill``: 2,048 tokens as 2 x 1024 in one step: median and best of the replayed step, the
  time of a step whose lengths were never seen before (inside a shape class that has a
  recording, and in a class seen for the very first time), flop fraction of the peak;
* ``roofline``: bytes a decode step has to read / its time, against the measured copy bandwidth;
* ``points``: decode tokens per second at batch 1, 8 and 64 and contexts 128, 512 and ~1014;
* ``fp32``: the headline step and the prefill in true 32-bit (no tensor cores);
* ``workloads``: GPT-2 medium (8 unequal prompts, 256 steps) and GPT-2 XL (64 prompts of 128
  tokens decoded to 1024) through ``Engine.generate``: time to the first token, decode and
  end-to-end tokens per second, bytes per step and their fraction of the copy bandwidth;
* ``clocks`` and ``gpu_launches``.

``python bench.py --designs`` is another measurement with a line of its own (the default
workload and its line stay as they are): with ``--design`` one of the other designs (Runesun,
Rizitar, Pinozen, Lulizen, Bumulix) beside GPT-2 or the closest design; by default the Runesun design (latent attention, routed experts)
beside GPT-2 at equal layer sizes (presets ``runesun-2k`` / ``gpt2-2k`` and ``runesun-1k`` /
``gpt2-1k``, random weights): decode steps at batch 8 and 64 and a 2 x 1024-token prefill, and
per kind of kernel the time inside a plainly launched step with its bytes, flops and fraction of
the measured roofline.

Every decode step reads all weights (247 MB in bf16) and the cache of the live requests,
far more than the 126 MB L2, so no L2 flush is needed between timed steps.  Model sizes come
from the package's presets (config files), none stands here.
"""
from __future__ import annotations

import argparse
import json
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

MODEL = "gpt2"                      # preset names (nimbus_infer_rs_b200/config/presets/)
OTHER_MODELS = ("gpt2-medium", "gpt2-xl")
CONTEXT = 1024
BATCH = 8
PREFILL_TOKENS = 2048
REFERENCE_DECODE_TOK_S = 35.1      # the reference's published CPU figure (README.md:25), batch 1
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
FP32_LANES_PER_SM = 128            # FMA lanes of an SM: nominal fp32 peak = SMs x lanes x 2 x clock


def load_peaks():
    p = ROOT / "MEASURED_PEAKS.json"
    if p.exists():
        try:
            d = json.loads(p.read_text())
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]),
                    "source": "measured"}
        except (OSError, ValueError, KeyError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.proc = None

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 6:
                self.samples.append(parts)

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        mhz, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for s in self.samples:
            try:
                mhz.append(int(s[0]))
                mx.append(int(s[1]))
            except ValueError:
                continue
            for n, v in zip(names, s[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        mhz.sort()
        return {"sm_mhz": mhz[len(mhz) // 2] if mhz else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(mhz)}


def prompts_for(batch, length, vocab, seed):
    import torch
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (length,), generator=g).tolist() for _ in range(batch)]


def time_decode(engine, batch, context, steps, warmup, seed=0):
    """Device time of exactly `steps` decode steps of `batch` sequences whose contexts end at
    `context`; returns (ms per step, kernel launches in the timed region, mean context)."""
    import torch
    from nimbus_infer_rs_b200.engine.decode import DecodeSession
    start = context - steps - warmup
    assert start >= 1, "steps + warmup must stay below the context length"
    V = engine.spec.vocab_size
    slots = [engine.alloc_slot() for _ in range(batch)]
    prompts = prompts_for(batch, start, V, seed)
    # prefill in chunks of at most 16 sequences to bound activation memory
    for i in range(0, batch, 16):
        engine.step([(s, p, []) for s, p in zip(slots[i:i + 16], prompts[i:i + 16])])
    session = DecodeSession(engine, slots, [p[-1] for p in prompts])
    for _ in range(warmup):
        session.step()
    torch.cuda.synchronize()
    launches0 = engine.ops.launches
    t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    t0.record()
    for _ in range(steps):
        session.step()
    t1.record()
    torch.cuda.synchronize()
    ms = t0.elapsed_time(t1) / steps
    launches = engine.ops.launches - launches0
    for s in slots:
        engine.free_slot(s)
    mean_ctx = start + warmup + (steps - 1) / 2.0 + 1
    return ms, launches, mean_ctx


def time_e2e(engine, batch, context, steps, warmup, seed=1):
    """Decode tokens per second through Engine.generate: per step the host hands the step's
    state over and reads the sampled tokens back.  Timed from the first sampled token of the
    timed window to the last, on the host clock."""
    import torch
    from nimbus_infer_rs_b200 import SamplingParams
    start = context - steps - warmup - 1
    prompts = prompts_for(batch, start, engine.spec.vocab_size, seed)
    stamps = {}

    def on_token(i, tok, step):
        if i == batch - 1 and step in (warmup, warmup + steps):
            torch.cuda.synchronize()
            stamps[step] = time.perf_counter()

    engine.generate(prompts, SamplingParams(max_new_tokens=warmup + steps + 1, temperature=0.0),
                    on_token=on_token, max_batch=batch)
    dt = stamps[warmup + steps] - stamps[warmup]
    return batch * steps / dt


def _timed_step(engine, entries):
    import torch
    torch.cuda.synchronize()
    t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    t0.record()
    engine.step(entries)
    t1.record()
    torch.cuda.synchronize()
    return t0.elapsed_time(t1)


def time_prefill(engine, n_seqs, length, reps=7):
    """One step of `n_seqs` prompts of `length` tokens, logits of each last token.  Returns
    milliseconds: median and best of `reps` replays of the recorded step (after two runs that
    warm up and record it), and the median over `reps` steps whose lengths were never seen
    before (a few tokens shorter each time: the step's shape class has a recording, its
    lengths are new)."""
    V = engine.spec.vocab_size

    def run(lengths, seed):
        slots = [engine.alloc_slot() for _ in lengths]
        prompts = [prompts_for(1, n, V, seed + i)[0] for i, n in enumerate(lengths)]
        ms = _timed_step(engine, [(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)])
        for s in slots:
            engine.free_slot(s)
        return ms

    run([length // 2 + 3] * n_seqs, 99)                # another class: loads the kernels
    first_sight = run([length] * n_seqs, 100)          # plain launches: the class is new
    run([length] * n_seqs, 101)                        # recorded here
    replays = [run([length] * n_seqs, 102 + r) for r in range(reps)]
    fresh = [run([length - 1 - 2 * r - i for i in range(n_seqs)], 200 + r) for r in range(reps)]
    return {"median": statistics.median(replays), "best": min(replays),
            "fresh_lengths": statistics.median(fresh), "first_sight": first_sight}


def model_flops_prefill(cfg, n_seqs, length):
    d, m, L, V = cfg.d_model, cfg.d_mlp, cfg.n_layers, cfg.vocab_size
    hq, hk = cfg.n_heads * cfg.head_dim, cfg.n_kv_heads * cfg.head_dim
    T = n_seqs * length
    linear = 2 * T * L * (d * (hq + 2 * hk) + hq * d + 2 * d * m)
    attn = n_seqs * L * 2 * 2 * cfg.n_heads * cfg.head_dim * (length * (length + 1) // 2)
    head = 2 * n_seqs * d * V
    return linear + attn + head


def kv_bytes_per_token(cfg, elt):
    return 2 * cfg.n_layers * cfg.n_kv_heads * cfg.head_dim * elt


def fp32_peak_tflops(clock_mhz):
    """Nominal: every SM retires `FP32_LANES_PER_SM` fused multiply-adds a clock."""
    import torch
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    return sms * FP32_LANES_PER_SM * 2 * clock_mhz * 1e6 / 1e12


def run_workload(engine, cfg, prompt_lens, n_new, hbm_gbs, windows=()):
    """A request list through Engine.generate (greedy, host tokens in and out every step).
    Timed on the host clock, the device waited for at each stamp: the prompts' step up to the
    first tokens, then the decode steps.  `windows`: contexts at which the decode rate of the
    32 steps around (or before) them is reported as well."""
    import torch
    from nimbus_infer_rs_b200 import SamplingParams
    V = engine.spec.vocab_size
    prompts = [prompts_for(1, n, V, 900 + i)[0] for i, n in enumerate(prompt_lens)]
    lead = min(range(len(prompts)), key=lambda i: len(prompts[i]))   # lives longest
    stamps = {}

    def on_token(i, tok, step):
        if i == lead:
            torch.cuda.synchronize()
            stamps[step] = time.perf_counter()

    torch.cuda.synchronize()
    t_start = time.perf_counter()
    out = engine.generate(prompts, SamplingParams(max_new_tokens=n_new, temperature=0.0),
                          on_token=on_token, max_batch=len(prompts))
    torch.cuda.synchronize()
    t_end = time.perf_counter()
    n_out = [len(o) for o in out]
    decoded = sum(n_out) - len(prompts)              # tokens that came from decode steps
    last = max(stamps)
    decode_s = stamps[last] - stamps[0]
    # bytes the decode steps had to read: every weight once a step, and the cache of each live
    # sequence (a sequence with n tokens out ran n - 1 decode steps)
    kvb = kv_bytes_per_token(cfg, 2)
    n_steps = max(n_out) - 1
    nbytes = n_steps * engine.model.weight_bytes()
    for plen, n in zip(prompt_lens, n_out):
        nbytes += kvb * sum(plen + t + 1 for t in range(n - 1))
    res = {"prompt_tokens": sum(prompt_lens), "prefill_ms": round((stamps[0] - t_start) * 1e3, 2),
           "decode_steps": n_steps, "decoded_tokens": decoded,
           "decode_tok_s": round(decoded / decode_s, 1),
           "e2e_tok_s": round(sum(n_out) / (t_end - t_start), 1),
           "decode_gb_per_step": round(nbytes / n_steps / 1e9, 3),
           "hbm_frac": round(nbytes / decode_s / 1e9 / hbm_gbs, 4)}
    for c in windows:
        hi = min(c - prompt_lens[lead], last)        # the step that brings the context to c
        lo = hi - 32
        if lo < 1:
            continue
        dt = stamps[hi] - stamps[lo]
        step_bytes = engine.model.weight_bytes() + len(prompts) * (c - 16) * kvb
        res[f"c{c}"] = {"tok_s": round(len(prompts) * 32 / dt, 1), "ms_per_step": round(dt / 32 * 1e3, 3),
                        "hbm_frac": round(step_bytes / (dt / 32) / 1e9 / hbm_gbs, 4)}
    return res


# ---------------------------------------------------------------------------------------------
# --designs: Runesun beside GPT-2 at equal layer sizes
# ---------------------------------------------------------------------------------------------
DESIGN_PAIRS = {"runesun": (("runesun-2k", "gpt2-2k"), ("runesun-1k", "gpt2-1k")),
                "rizitar": (("rizitar-2k", "gpt2-2k"), ("rizitar-1k", "gpt2-1k")),
                # beside the closest design of the library: recurrent layers among attention layers
                "pinozen": (("pinozen-2k", "rizitar-2k"), ("pinozen-1k", "rizitar-1k")),
                # beside the closest design of the library: sublayers between two norms, attention
                # with normed and rotated queries and keys over a window, routed experts
                "lulizen": (("lulizen-2k", "rizitar-2k"), ("lulizen-1k", "rizitar-1k")),
                # beside the two closest designs: Lulizen's masked attention over shared key heads
                # and Runesun's attention over a latent
                "bumulix": (("bumulix-2k", "lulizen-2k", "runesun-2k"),
                            ("bumulix-1k", "lulizen-1k", "runesun-1k")),
                # beside the two closest designs: Lulizen's masked attention and routed experts
                # with a shared one, Rizitar's delta rule and per-token input
                "zorulix": (("zorulix-2k", "lulizen-2k", "rizitar-2k"),
                            ("zorulix-1k", "lulizen-1k", "rizitar-1k"))}


class OpTimer:
    """Times every call into the kernel library during plainly launched steps (CUDA events on
    the stream around each call) and notes the bytes a call has to move and its flops, from the
    tensors it is given.  Kernels of a kind are added up."""

    KINDS = ("linear", "layernorm", "rmsnorm", "attention", "attention_latent", "latent_append",
             "head_linear", "moe_route", "moe_group", "moe_linear", "moe_combine", "embed_pos",
             "rms_add", "act_rows", "gather_mul", "qk_norm_rope_append", "pool_blocks",
             "attention_pooled", "delta_rule", "conv_rope_append", "conv_act", "attention_capped",
             "selective_scan", "linear_attention", "rmsnorm_gated", "rms_pair_add", "glu_rows",
             "cast_cols", "embed_hashed", "ln_add", "qkv_norm_rope_append",
             "attention_masked", "moe_route_sigmoid", "attention_differential",
             "latent_rope_append", "streams", "softcap_rows", "gated_delta", "scaled_pair_add")

    def __init__(self, ops):
        import torch
        self.torch, self.ops, self.records, self._orig = torch, ops, [], {}
        self._depth = 0
        # written before every timed call: it empties the L2 (larger than its 126 MB), and while
        # the GPU is busy with it the host gets the call's launches queued, so that the events
        # see the kernels' time and not the host's
        self.flush = torch.empty(256 << 20, dtype=torch.int8, device="cuda")
        for kind in self.KINDS:
            if hasattr(ops, kind):
                self._orig[kind] = getattr(ops, kind)
                setattr(ops, kind, self._wrap(kind, self._orig[kind]))

    def close(self):
        for kind in self._orig:
            delattr(self.ops, kind)

    def _wrap(self, kind, fn):
        torch = self.torch

        def call(*a, **kw):
            if self._depth:      # an op that hands on to another one is timed once, as itself
                return fn(*a, **kw)
            t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            self.flush.zero_()
            t0.record()
            self._depth += 1
            try:
                fn(*a, **kw)
            finally:
                self._depth -= 1
            t1.record()
            self.records.append((kind, self._label(kind, a, kw), t0, t1, *self._work(kind, a, kw)))
        return call

    @staticmethod
    def _nbytes(*ts):
        return sum(t.numel() * t.element_size() for t in ts if t is not None)

    def _label(self, kind, a, kw):
        if kind == "linear":
            return f"linear {a[1].shape[0]}x{a[1].shape[1]}"
        if kind == "moe_linear":
            return "moe_linear gate+up" if a[5] is not None else (
                "moe_linear up" if a[1] is not None else "moe_linear down")
        if kind == "attention_masked" and self._value_size(a[2], a[3]) != a[2].head_dim:
            return f"attention_masked, keys of {a[2].head_dim}, values of {self._value_size(a[2], a[3])}"
        return kind

    @staticmethod
    def _value_size(keys, values):
        return keys.value_size if values is keys else values.head_dim

    def _work(self, kind, a, kw):
        """(bytes, flops) of one call."""
        nb = self._nbytes
        if kind == "linear":
            x, w, bias, out = a[0], a[1], a[2], a[3]
            return nb(w, out) + x.shape[0] * w.shape[1] * w.element_size(), 2 * x.shape[0] * w.shape[0] * w.shape[1]
        if kind in ("attention", "attention_latent"):
            if kind == "attention":
                q, lay, kv, heads = a[0], a[2], a[3], a[4]
                per_key, planes = kv.n_kv_heads * kv.head_dim, 2
                width = heads * kv.head_dim
            else:
                q, lay, kv, heads, out = a[0], a[1], a[2], a[3], a[5]
                keys = sum(p + n for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
                pairs = sum(n * p + n * (n + 1) // 2 for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
                return keys * kv.head_dim * kv.k.element_size() + nb(q, out), \
                    2 * pairs * (q.shape[1] + out.shape[1])
            elt = kv.k.element_size()
            keys = sum(p + n for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            pairs = sum(n * p + n * (n + 1) // 2 for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            return keys * per_key * planes * elt + 2 * lay.n_tokens * width * elt, 4 * pairs * width
        if kind == "head_linear":
            x, w, out, lay = a[0], a[2], a[3], a[4]
            return nb(w, out) + lay.n_rows * w.shape[0] * w.shape[2] * x.element_size(), \
                2 * lay.n_rows * w.shape[0] * w.shape[1] * w.shape[2]
        if kind == "moe_linear":
            x, offsets, w, w2, out = a[0], a[3], a[4], a[5], a[6]
            off = offsets.cpu()
            used = int(((off[1:] - off[:-1]) > 0).sum())
            sets = 2 if w2 is not None else 1
            pairs = int(off[-1])
            return used * sets * w.shape[1] * w.shape[2] * w.element_size() + nb(out) + \
                pairs * w.shape[2] * x.element_size(), 2 * pairs * sets * w.shape[1] * w.shape[2]
        if kind in ("layernorm", "rmsnorm"):
            out = a[4] if kind == "layernorm" else a[3]
            return 4 * out.numel() + nb(out), 0
        if kind == "moe_combine":
            return nb(a[0], a[4] if len(a) > 4 else None) + 2 * nb(a[3]), 0
        if kind == "scaled_pair_add":
            return nb(a[0], a[2], a[7]) + 2 * nb(a[4]), 0
        if kind == "gated_delta":
            taps, lay, heads, kv_heads, d, dv, out = a[3], a[15], *a[17:22]
            # q, k, v, the logits of rate, decay and gate per token, the state of every
            # sequence in and out; per token and head 4 d dv multiply-adds on the CUDA cores
            per_token = 2 * kv_heads * d + heads * (2 * dv + d + 1)
            state = heads * d * dv + max(int(taps) - 1, 0) * (2 * kv_heads * d + heads * dv)
            return lay.n_tokens * per_token * 4 + nb(out) + 2 * lay.n_seqs * state * 4, \
                2 * 4 * lay.n_tokens * heads * d * dv
        if kind in ("rms_add", "ln_add"):
            return nb(a[0], a[6], a[7]) + 2 * nb(a[3]), 0
        if kind == "embed_hashed":
            return a[4].numel() * (4 + 2 * a[1].element_size()), 0
        if kind == "moe_route_sigmoid":
            return nb(a[0]) + 2 * nb(a[12]), 0
        if kind == "qkv_norm_rope_append":
            lay, ks, vs, heads, q = a[10], a[11], a[12], a[13], a[15]
            kv = ks.n_kv_heads * (ks.head_dim + self._value_size(ks, vs)) if a[16] else 0
            return lay.n_tokens * (4 * (heads * ks.head_dim + kv) + kv * ks.k.element_size()) + nb(q), 0
        if kind == "attention_masked":
            q, lay, ks, vs, heads, out = a[0], a[1], a[2], a[3], a[4], a[6]
            window, keep, block = (list(a[9:12]) + [0, 0, 0])[:3] if len(a) > 9 else (
                kw.get("window", 0), kw.get("keep_first", 0), kw.get("chunk", 0))
            elt = ks.k.element_size()

            def first(i):       # the first key of the run that ends at position i
                return (i // block) * block if block else (max(0, i + 1 - window) if window else 0)
            pairs = sum(i + 1 - first(i) + (min(keep, first(i)) if window else 0)
                        for p, n in zip(lay.seq_pos0_host, lay.seq_lens) for i in range(p, p + n))
            # every sequence's keys once (neighbouring rows share them), queries, outputs
            keys = sum(p + n - first(p) + (min(keep, first(p)) if window else 0)
                       for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            both = ks.head_dim + self._value_size(ks, vs)
            return keys * ks.n_kv_heads * both * elt + nb(q, out), 2 * pairs * heads * both
        if kind == "attention_differential":
            q, lay, ks, vs, heads, out, window = a[0], a[1], a[2], a[3], a[4], a[5], a[7]

            def first(i):
                return max(0, i + 1 - window) if window else 0
            pairs = sum(i + 1 - first(i) for p, n in zip(lay.seq_pos0_host, lay.seq_lens)
                        for i in range(p, p + n))
            keys = sum(p + n - first(p) for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            # two maps of half a key each, both over the whole values
            return keys * ks.n_kv_heads * (ks.head_dim + vs.head_dim) * ks.k.element_size() + nb(q, out), \
                2 * pairs * heads * (ks.head_dim + 2 * vs.head_dim)
        if kind == "latent_rope_append":
            rot, q, heads, lay, kv = a[5], a[8], a[11], a[12], a[13]
            return lay.n_tokens * ((kv.head_dim + heads * rot) * (4 + kv.k.element_size())), 0
        if kind == "streams":
            x, S, spread = a[0], a[1], a[2]
            y = kw["write"][0] if kw.get("write") else None
            return nb(x, y, kw.get("into"), kw.get("total"), kw.get("out") if kw.get("read") else None), 0
        if kind == "softcap_rows":
            return 2 * nb(a[0]), 0
        if kind == "act_rows":
            return 4 * a[4].numel() + nb(a[4]), 0
        if kind == "gather_mul":
            return nb(a[0], a[3]) + a[3].numel() * a[1].element_size(), 0
        if kind == "qk_norm_rope_append":
            lay, kv, heads, q = a[9], a[10], a[11], a[12]
            width = (heads + kv.n_kv_heads) * kv.head_dim
            return lay.n_tokens * (4 * width + 2 * kv.n_kv_heads * kv.head_dim * kv.k.element_size()) + nb(q), 0
        if kind == "attention_pooled":
            q, lay, kv, heads, window, pool = a[0], a[1], a[2], a[4], a[8], a[9]
            elt, per_key = kv.k.element_size(), kv.n_kv_heads * kv.head_dim
            width = heads * kv.head_dim

            def seen(i):        # entries position i sees: its window and the blocks before it
                w = min(i + 1, window) if window else i + 1
                return w + (max(0, (i + 1 - window) // pool) if window and pool else 0)
            pairs = sum(seen(i) for p, n in zip(lay.seq_pos0_host, lay.seq_lens) for i in range(p, p + n))
            # every sequence's window and blocks once (a row's neighbours share them), queries, outputs
            keys = sum(seen(p + n - 1) + (n - 1 if window else 0) for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            return keys * per_key * 2 * elt + 2 * lay.n_tokens * width * elt, 4 * pairs * width
        if kind == "conv_rope_append":
            w, taps, lay, ks, vs, heads, q = a[2], a[3], a[7], a[8], a[9], a[10], a[12]
            ch = heads * ks.head_dim + ks.n_kv_heads * (ks.head_dim + vs.head_dim)
            # the projected rows once, the cached keys and values, the queries, the state in and out
            return lay.n_tokens * (4 * ch + (ch - heads * ks.head_dim) * ks.k.element_size()) + nb(q, w) + \
                2 * lay.n_seqs * max(int(taps) - 1, 0) * ch * 4, 0
        if kind == "conv_act":
            w, taps, lay, out, out_act = a[2], a[4], a[7], a[8], (a[9] if len(a) > 9 else None)
            return 4 * out.numel() + nb(out, out_act, w) + 2 * lay.n_seqs * max(int(taps) - 1, 0) * out.shape[1] * 4, 0
        if kind == "attention_capped":
            q, lay, ks, vs, heads, out = a[0], a[1], a[2], a[3], a[4], a[6]
            elt = ks.k.element_size()
            keys = sum(p + n for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            pairs = sum(n * p + n * (n + 1) // 2 for p, n in zip(lay.seq_pos0_host, lay.seq_lens))
            return keys * ks.n_kv_heads * (ks.head_dim + vs.head_dim) * elt + nb(q, out), \
                2 * pairs * heads * (ks.head_dim + vs.head_dim)
        if kind == "selective_scan":
            x, low, dt_lin, lay, n_state, out = a[0], a[1], a[4], a[11], a[12], a[13]
            inner = x.shape[1]
            # inputs, step sizes and gates per token, B and C, the state of every sequence in and
            # out; per token, channel and state number an exponential and three multiply-adds
            return lay.n_tokens * (3 * inner + 2 * n_state) * 4 + nb(out) + 2 * lay.n_seqs * inner * n_state * 4, \
                2 * 4 * lay.n_tokens * inner * n_state
        if kind == "linear_attention":
            lay, heads, d, dv, out = a[7], a[8], a[9], a[10], a[11]
            return lay.n_tokens * heads * (2 * d + dv) * 4 + nb(out) + 2 * lay.n_seqs * heads * d * dv * 4, \
                2 * 2 * lay.n_tokens * heads * d * dv
        if kind == "rmsnorm_gated":
            return 2 * 4 * a[5].numel() + nb(a[5]), 0
        if kind == "rms_pair_add":
            return nb(a[0], a[2], kw.get("out_next", a[9] if len(a) > 9 else None)) + 2 * nb(a[6]), 0
        if kind == "glu_rows":
            return 2 * 4 * a[4].numel() + nb(a[4]), 0
        if kind == "cast_cols":
            return nb(a[0]) + a[0].numel() * a[1].element_size(), 0
        if kind == "delta_rule":
            fused, lay, state, heads, dim, out = a[0], a[12], a[13], a[14], a[15], a[16]
            hd = heads * dim
            # five fp32 vectors and the decay's logits per token, the state of every sequence in
            # and out; per token and head 6 dim^2 multiply-adds on the CUDA cores
            return lay.n_tokens * 6 * hd * 4 + nb(out) + 2 * lay.n_seqs * hd * dim * 4, \
                2 * 3 * lay.n_tokens * hd * dim
        return 0, 0

    def table(self, peaks):
        self.torch.cuda.synchronize()
        rows = {}
        for kind, label, t0, t1, nbytes, flops in self.records:
            r = rows.setdefault(label, {"calls": 0, "ms": 0.0, "bytes": 0, "flops": 0})
            r["calls"] += 1
            r["ms"] += t0.elapsed_time(t1)
            r["bytes"] += nbytes
            r["flops"] += flops
        for r in rows.values():
            ideal_ms = max(r["bytes"] / (peaks["hbm_gbs"] * 1e6), r["flops"] / (peaks["bf16_tflops"] * 1e9))
            r["us_per_call"] = round(1e3 * r["ms"] / r["calls"], 2)
            r["of_roofline"] = round(ideal_ms / r["ms"], 4) if r["ms"] > 0 and ideal_ms > 0 else None
            r["bound"] = "hbm" if r["bytes"] / (peaks["hbm_gbs"] * 1e6) >= r["flops"] / (peaks["bf16_tflops"] * 1e9) else "tensor"
            r["ms"] = round(r["ms"], 4)
        self.records = []
        return rows


def profile_ops(engine, peaks, batch, context, prefill):
    """Per kind of kernel: a decode step of `batch` sequences at `context`, and a prompt step of
    `prefill` = (sequences, length), both launched plainly with events around every call."""
    import torch
    V = engine.spec.vocab_size
    graphs, engine.step_graphs = engine.step_graphs, None
    timer = OpTimer(engine.ops)
    out = {}
    try:
        slots = [engine.alloc_slot() for _ in range(batch)]
        for i in range(0, batch, 16):
            engine.step([(s, p, []) for s, p in zip(slots[i:i + 16], prompts_for(len(slots[i:i + 16]), context - 4, V, 5 + i))])
        nxt = prompts_for(3, batch, V, 4)       # every sequence goes on with a token of its own
        for k in range(2):
            engine.step([(s, [tok], [0]) for s, tok in zip(slots, nxt[k])])
        timer.records = []
        torch.cuda.synchronize()
        engine.step([(s, [tok], [0]) for s, tok in zip(slots, nxt[2])])
        out["decode"] = timer.table(peaks)
        for s in slots:
            engine.free_slot(s)
        n_seqs, length = prefill
        for rep in range(2):
            slots = [engine.alloc_slot() for _ in range(n_seqs)]
            timer.records = []
            torch.cuda.synchronize()
            engine.step([(s, p, [length - 1]) for s, p in zip(slots, prompts_for(n_seqs, length, V, 6 + rep))])
            table = timer.table(peaks)
            for s in slots:
                engine.free_slot(s)
        out["prefill"] = table
    finally:
        timer.close()
        engine.step_graphs = graphs
    return out


def compare_designs(args, peaks):
    import torch
    from nimbus_infer_rs_b200 import Engine
    results = []
    launches = 0
    with ClockSampler() as clocks:
        for pair in DESIGN_PAIRS[args.design]:
            entry = {}
            for name in pair:
                engine = Engine.random(name, seed=0, dtype="bfloat16", cache_tokens=66 * CONTEXT)
                r = {"weight_mb": round(engine.model.weight_bytes() / 2 ** 20, 1)}
                for batch in (8, 64):
                    ms, n, _ = time_decode(engine, batch, CONTEXT, args.steps, args.warmup)
                    launches += n
                    r[f"decode_b{batch}_ms"] = round(ms, 4)
                    r[f"decode_b{batch}_tok_s"] = round(batch / (ms * 1e-3), 1)
                pre = time_prefill(engine, PREFILL_TOKENS // CONTEXT, CONTEXT, reps=5)
                r["prefill_2x1024_ms"] = round(pre["median"], 4)
                r["prefill_tok_s"] = round(PREFILL_TOKENS / (pre["median"] * 1e-3), 1)
                r["kernels"] = profile_ops(engine, peaks, 8, CONTEXT, (PREFILL_TOKENS // CONTEXT, CONTEXT))
                entry[name] = r
                del engine
                torch.cuda.empty_cache()
            results.append(entry)
    print(json.dumps({"designs": results, "dtype": "bf16", "data": "synthetic", "steps": args.steps,
                      "warmup": args.warmup, "gpu_launches": launches, "clocks": clocks.summary(),
                      "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops")},
                      "config": {"decode_context": CONTEXT, "prefill": "2 x 1024 tokens",
                                 "l2": "decode and prefill steps read the model's weights, larger "
                                       "than L2; the per-kernel profile writes 256 MB before every "
                                       "timed call"}}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--dtype", default="bf16", choices=["bf16", "fp32"])
    ap.add_argument("--no-points", action="store_true", help="skip the other batch sizes and contexts")
    ap.add_argument("--no-fp32", action="store_true", help="skip the 32-bit figures")
    ap.add_argument("--no-workloads", action="store_true", help="skip the medium and XL workloads")
    ap.add_argument("--only", default="all", choices=["all", "decode", "prefill"],
                    help="measure one phase only (for profiling); prints a reduced line")
    ap.add_argument("--batch", type=int, default=BATCH, help="batch of the decode step")
    ap.add_argument("--context", type=int, default=CONTEXT, help="with --only decode: context the steps end at")
    ap.add_argument("--model", default=MODEL, choices=[MODEL, *OTHER_MODELS],
                    help="layer sizes (a preset); other than the default only with --only")
    ap.add_argument("--designs", action="store_true",
                    help="instead of the headline: another design beside GPT-2 at equal layer sizes "
                         "(decode, prefill, per-kernel roofline fractions)")
    ap.add_argument("--design", default="runesun", choices=sorted(DESIGN_PAIRS),
                    help="with --designs: which design stands beside GPT-2")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference is a Rust crate (Cargo.toml, no Python package); there is "
                          "no Rust toolchain on this box, so it cannot be built or installed"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU only (asked for {args.gpus}): this library has no "
              "multi-GPU path")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch
    from nimbus_infer_rs_b200 import Engine
    from nimbus_infer_rs_b200.config import load_preset

    peaks = load_peaks()
    if args.designs:
        return compare_designs(args, peaks)
    dtype = "bfloat16" if args.dtype == "bf16" else "float32"
    if args.model != MODEL and args.only == "all":
        print("--model other than gpt2 needs --only decode or --only prefill")
        return 2
    _, cfg, _ = load_preset(args.model)
    cache_tokens = max(64, args.batch if args.only == "decode" else 64) * CONTEXT + 64
    engine = Engine.random(args.model, seed=0, dtype=dtype, cache_tokens=cache_tokens)
    elt = 2 if dtype == "bfloat16" else 4

    if args.only == "prefill":
        pre = time_prefill(engine, PREFILL_TOKENS // CONTEXT, CONTEXT, reps=8)
        flops = model_flops_prefill(cfg, PREFILL_TOKENS // CONTEXT, CONTEXT)
        print(json.dumps({"only": "prefill", "model": args.model, "dtype": args.dtype,
                          "ms": round(pre["median"], 4), "ms_best": round(pre["best"], 4),
                          "fresh_lengths_ms": round(pre["fresh_lengths"], 4),
                          "first_sight_ms": round(pre["first_sight"], 4),
                          "tokens_per_s": round(PREFILL_TOKENS / (pre["median"] * 1e-3), 1),
                          "tflops": round(flops / (pre["median"] * 1e-3) / 1e12, 1)}))
        return 0
    if args.only == "decode":
        ms, launches, mean_ctx = time_decode(engine, args.batch, args.context, args.steps, args.warmup)
        nbytes = engine.model.weight_bytes() + args.batch * mean_ctx * kv_bytes_per_token(cfg, elt)
        print(json.dumps({"only": "decode", "model": args.model, "dtype": args.dtype,
                          "batch": args.batch, "context": args.context, "ms_per_step": round(ms, 4),
                          "tokens_per_s": round(args.batch * 1000.0 / ms, 1),
                          "gb_per_s": round(nbytes / (ms * 1e-3) / 1e9, 1),
                          "gpu_launches": launches}))
        return 0

    n_pre = PREFILL_TOKENS // CONTEXT
    pre_flops = model_flops_prefill(cfg, n_pre, CONTEXT)
    # clocks and throttle reasons are sampled while all of the measurements below run
    with ClockSampler() as clocks:
        ms, launches, mean_ctx = time_decode(engine, BATCH, CONTEXT, args.steps, args.warmup)
        value = BATCH * 1000.0 / ms
        step_bytes = engine.model.weight_bytes() + BATCH * mean_ctx * kv_bytes_per_token(cfg, elt)
        achieved = step_bytes / (ms * 1e-3) / 1e9

        e2e = time_e2e(engine, BATCH, CONTEXT, args.steps, args.warmup)

        pre = time_prefill(engine, n_pre, CONTEXT)
        time.sleep(0.12)
    clock_summary = clocks.summary()
    fp32_peak = fp32_peak_tflops(clock_summary.get("sm_max_mhz") or 1965)
    peak_flops = peaks["bf16_tflops"] * 1e12 if dtype == "bfloat16" else fp32_peak * 1e12
    prefill = {"value": round(PREFILL_TOKENS / (pre["median"] * 1e-3), 1), "tokens": PREFILL_TOKENS,
               "ms": round(pre["median"], 4),
               "frac": round(pre_flops / (pre["median"] * 1e-3) / peak_flops, 4),
               "ms_best": round(pre["best"], 4), "fresh_lengths_ms": round(pre["fresh_lengths"], 4),
               "first_sight_ms": round(pre["first_sight"], 4)}
    # the other batch sizes and contexts run without the clock sampler beside them: a step at
    # batch 1 is short enough for the sampler's process to show in it
    points = {}
    if not args.no_points:
        for b in (1, 64):
            pms, _, _ = time_decode(engine, b, CONTEXT, args.steps, args.warmup, seed=b)
            points[f"decode_b{b}"] = round(b * 1000.0 / pms, 1)
        for c in (128, 512):
            for b in (1, BATCH, 64):
                st = min(args.steps, c - args.warmup - 8)
                pms, _, _ = time_decode(engine, b, c, st, args.warmup, seed=b + c)
                points[f"decode_b{b}_c{c}"] = round(b * 1000.0 / pms, 1)

    fp32 = None
    if not args.no_fp32 and dtype == "bfloat16":
        del engine
        torch.cuda.empty_cache()
        e32 = Engine.random(MODEL, seed=0, dtype="float32", cache_tokens=16 * CONTEXT + 64)
        ms32, _, ctx32 = time_decode(e32, BATCH, CONTEXT, 16, 3)
        b32 = e32.model.weight_bytes() + BATCH * ctx32 * kv_bytes_per_token(cfg, 4)
        p32 = time_prefill(e32, n_pre, CONTEXT, reps=3)
        fp32 = {"decode_b8_tok_s": round(BATCH * 1000.0 / ms32, 1), "decode_ms_per_step": round(ms32, 4),
                "decode_hbm_frac": round(b32 / (ms32 * 1e-3) / 1e9 / peaks["hbm_gbs"], 4),
                "prefill_ms": round(p32["median"], 3),
                "prefill_tok_s": round(PREFILL_TOKENS / (p32["median"] * 1e-3), 1),
                "prefill_frac": round(pre_flops / (p32["median"] * 1e-3) / (fp32_peak * 1e12), 4),
                "peak_tflops": round(fp32_peak, 1)}
        del e32
        engine = None

    workloads = {}
    if not args.no_workloads and dtype == "bfloat16":
        engine = None
        torch.cuda.empty_cache()
        # GPT-2 medium: 8 unequal prompts, 256 decode steps; a sequence that reaches the end of
        # the context stops earlier
        _, mcfg, _ = load_preset("gpt2-medium")
        em = Engine.random("gpt2-medium", seed=0, dtype="bfloat16", cache_tokens=8 * CONTEXT + 64)
        lens = [32, 160, 288, 416, 544, 672, 800, 1000]
        # (a run of another, larger shape class first: it loads the kernels and leaves the
        # allocator with blocks that are large enough; the timed run is then the first sight of
        # its own shape class, as a fresh request list is)
        run_workload(em, mcfg, [min(l + 40, 1016) for l in lens], 4, peaks["hbm_gbs"])
        workloads["medium"] = run_workload(em, mcfg, lens, 257, peaks["hbm_gbs"])
        del em
        torch.cuda.empty_cache()
        # GPT-2 XL: 64 prompts of 128 tokens, decoded to the end of the context
        _, xcfg, _ = load_preset("gpt2-xl")
        ex = Engine.random("gpt2-xl", seed=0, dtype="bfloat16", cache_tokens=64 * CONTEXT + 64)
        run_workload(ex, xcfg, [96] * 64, 4, peaks["hbm_gbs"])
        workloads["xl"] = run_workload(ex, xcfg, [128] * 64, CONTEXT - 128, peaks["hbm_gbs"],
                                       windows=(256, 512, 1024))
        del ex

    b1 = points.get("decode_b1")
    out = {
        "metric": "decode tok/s, GPT-2 124M, batch 8, context 1024", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": round(b1 / REFERENCE_DECODE_TOK_S, 1) if b1 else None, "dtype": args.dtype,
        "data": "synthetic: random-init weights N(0,0.02), uniform random token ids",
        "config": {"model": "gpt2-124M", "n_layer": cfg.n_layers, "n_layer_model": 12,
                   "n_embd": cfg.d_model, "n_head": cfg.n_heads, "head_dim": cfg.head_dim,
                   "n_inner": cfg.d_mlp, "vocab_size": cfg.vocab_size,
                   "n_positions": cfg.max_seq_len, "tied_head": cfg.tie_embeddings,
                   "global_batch": BATCH, "seq_len": CONTEXT,
                   "decode_context_mean": round(mean_ctx, 1), "parallelism": "single-gpu",
                   "l2": "inputs larger than L2 (weights + cache read per step)",
                   "peaks": peaks["source"] + "; fp32: nominal SMs x 128 FMA lanes x 2 x max clock",
                   "baseline": "vs_baseline = batch-1 decode / the reference's CPU batch-1 decode, "
                               "35.1 tok/s (README.md:25)",
                   "medium": "gpt2-medium L24 d1024 H16 m4096: 8 prompts of 32..1000 tokens, 256 steps",
                   "xl": "gpt2-xl L48 d1600 H25 m6400: 64 prompts of 128 tokens decoded to 1024"},
        "e2e": {"value": round(e2e, 1), "unit": "tokens/s",
                "h2d_bytes_per_step": BATCH * 4, "d2h_bytes_per_step": BATCH * 4},
        "gpu_launches": launches,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"],
                     "unit": "GB/s", "frac": round(achieved / peaks["hbm_gbs"], 4)},
        "points": points,
        "fp32": fp32,
        "workloads": workloads,
        "clocks": clock_summary,
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
