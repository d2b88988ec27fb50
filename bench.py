"""Benchmark of the decode step (and of a 2,048-token prefill) of the
Qwen2.5-7B shape with random bfloat16 weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers L]
                    [--shape qwen2.5-7b|qwen2.5-0.5b|qwen2.5-32b] [--workload equal|unequal]

Prints ONE JSON line.  `value` is decoded tokens per second at the default
batch, timed on the device with CUDA events around K decode steps that are
launched back to back (tokens are given, nothing waits for the host).  `e2e`
is the same through the Python entry point `Engine.generate()`: prompts go in
as host token ids and every step's token ids come back to the host (the loop
reads them one step late, while the device runs the next step); it runs for
at least 128 timed steps whatever K is, after warm-up steps as the device-timed
run has them (`e2e.steps`, `e2e.warmup`).  `prefill`
is one step over a 2,048-token prompt (timed the second time: like every single prompt from position 0 it then
replays the graph captured the first time, the same kernels without the host's launches between them); `roofline` relates the decode step's
necessary bytes (every weight it uses once, the cache of the live sequences)
to its time; `points` hold decode at batch 1 and 64, device-timed and end to
end, and the time to the first token of a 32- and a 2,048-token prompt through
`Engine.generate()` (`ttft_ms_p32`, `ttft_ms_p2048`); `kernels` holds the device time of one decode step and of the prefill by
class of kernel (launched one by one behind a head start of other work, with
events between the classes) and what each class achieves of the measured
peak.  `--workload unequal` is the second benchmark configuration: a batch of
64 prompts with seeded lengths uniform in 64..4,096, prefilled in ONE step,
then 256 decode steps.  Peaks come from MEASURED_PEAKS.json beside this file
if it exists, else from an earlier measurement on the same kind of machine
(6.65 TB/s, 1.59 PFLOP/s).

`--design zodosun|rirudra|pavisun|furesun|gokapel|safurax [--sizes 1k,2k,4k] [--prompt 2048]` is another program: the named decoder beside the Qwen2
decoder of the same width, depth, heads, feed-forward and vocabulary (random weights, bfloat16): device time of a
prompt, of decode steps at batch 8 and 64, and the time by class of kernel with what the attention and scan
kernels reach of their rooflines, as one JSON line of its own (`--design rirudra` also runs the Zodosun decoder,
whose scans are the like kernels of its own; `--design pavisun` runs the Pavisun decoder and the Qwen2 decoder only;
`--design furesun` runs the Furesun, Rirudra and Qwen2 decoders; `--design gokapel` the Gokapel, Rirudra, Pavisun and
Qwen2 decoders; `--design safurax` the Safurax, Furesun and Qwen2 decoders).  The default workload and its line are untouched.

The reference arm (`--impl reference`) cannot run here: the reference is a
Rust workspace and no Rust toolchain is installed, so it prints its
`unavailable` line.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks() -> tuple[dict, str]:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            with open(path) as f:
                d = json.load(f)
            out = dict(FALLBACK_PEAKS)
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                if k in d and d[k]:
                    out[k] = float(d[k])
            return out, "measured"
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    NAMES = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]

    def __init__(self):
        self.samples: list[list[str]] = []
        self._stop = threading.Event()
        self._t = None

    def _run(self):
        while not self._stop.is_set():
            try:
                out = subprocess.run(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                      "--format=csv,noheader,nounits"], capture_output=True, text=True, timeout=5)
                if out.returncode == 0 and out.stdout.strip():
                    self.samples.append([x.strip() for x in out.stdout.strip().splitlines()[0].split(",")])
            except Exception:
                pass
            self._stop.wait(0.1)

    def __enter__(self):
        self._t = threading.Thread(target=self._run, daemon=True)
        self._t.start()
        return self

    def __exit__(self, *a):
        self._stop.set()
        self._t.join(timeout=6)

    def summary(self) -> dict:
        mhz = [int(s[0]) for s in self.samples if s and s[0].isdigit()]
        mx = [int(s[1]) for s in self.samples if len(s) > 1 and s[1].isdigit()]
        reasons = sorted({n for s in self.samples for n, v in zip(self.NAMES, s[2:]) if v.lower().startswith("active")})
        return {"sm_mhz": int(statistics.median(mhz)) if mhz else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(mhz)}


def model_numbers(cfg: dict, n_layers: int) -> dict:
    """Parameters in matrix products per layer, bytes a decode step must read,
    flops of a step, and the same by class of kernel."""
    H, nh, nkv = cfg["hidden_size"], cfg["num_attention_heads"], cfg["num_key_value_heads"]
    hd, I, V = cfg["head_dim"], cfg["intermediate_size"], cfg["vocab_size"]
    per_class = {"qkv": (nh + 2 * nkv) * hd * H, "o": H * nh * hd, "gate_up": 2 * I * H, "down": I * H}
    layer_mm = sum(per_class.values())
    layer_small = (nh + 2 * nkv) * hd + 2 * H
    weight_bytes = 2 * (n_layers * (layer_mm + layer_small) + V * H + H)     # the embedding table is not read
    kv_bytes_per_token = 2 * nkv * hd * 2 * n_layers
    return {"layer_mm": layer_mm, "weight_bytes": weight_bytes, "kv_bytes_per_token": kv_bytes_per_token,
            "head_mm": V * H, "attn_flops_per_key": 4 * nh * hd * n_layers,
            "class_params": {k: v * n_layers for k, v in per_class.items()}}


CLASSES = ["embed", "norms", "qkv", "rotary", "attention", "o", "gate_up", "down", "head", "sampler"]


def class_table(totals_us: dict, prefix: str, nums: dict, pk: dict, *, tokens: int, cached_tokens: float,
                wanted_rows: int, decode: bool, attn_flops: float = 0.0) -> dict:
    """Flat `kernels` entries of one step: microseconds per class, and for the classes with a roofline what
    they reach of it: GB/s over the measured copy bandwidth for a decode step (weights once, the cache),
    TFLOP/s over the measured bf16 peak for a prompt."""
    out = {}
    for c in CLASSES:
        us = totals_us.get(c)
        if us is None:
            continue
        out[f"{prefix}.{c}.us"] = round(us, 1)
        params = nums["class_params"].get(c) if c != "head" else nums["head_mm"]
        if decode:
            nbytes = 2 * params if params else (cached_tokens * nums["kv_bytes_per_token"] if c == "attention" else 0)
            if nbytes:
                gbs = nbytes / (us * 1e-6) / 1e9
                out[f"{prefix}.{c}.gbs"] = round(gbs, 1)
                out[f"{prefix}.{c}.frac"] = round(gbs / pk["hbm_gbs"], 3)
        else:
            rows = wanted_rows if c == "head" else tokens
            flops = 2 * rows * params if params else (attn_flops if c == "attention" else 0)
            if flops and c != "head":
                tf = flops / (us * 1e-6) / 1e12
                out[f"{prefix}.{c}.tflops"] = round(tf, 1)
                out[f"{prefix}.{c}.frac"] = round(tf / pk["bf16_tflops"], 3)
    out[f"{prefix}.sum.us"] = round(sum(v for k, v in totals_us.items() if k in CLASSES), 1)
    return out


def timed_by_class(run, reps: int = 3) -> dict:
    """Median device time by class of `run()` (a step launched kernel by kernel).  The device is first given
    some tens of milliseconds of other work, so that the host has launched the whole step before the device
    reaches it and the events between the classes see the kernels back to back, not the host's pace."""
    import torch
    from tq_kv_b200 import kernels
    a = torch.randn(8192, 8192, device="cuda", dtype=torch.bfloat16)
    runs = []
    for _ in range(reps):
        torch.cuda.synchronize()
        tl = kernels.Timeline()
        for _ in range(48):
            torch.mm(a, a)
        kernels._lib.timeline = tl
        try:
            tl.mark("start")
            run()
        finally:
            kernels._lib.timeline = None
        runs.append(tl.totals())
    return {k: statistics.median(r.get(k, 0.0) for r in runs) for k in runs[0]}


# ---- --design zodosun: the Zodosun decoder beside the Qwen2 decoder of equal size ---------------------------------
DESIGN_SIZES = {          # width, feed-forward width, layers (delta, delta, side-by-side, delta), vocabulary
    "1k": (1024, 2816, 4, 32000),
    "2k": (2048, 5632, 4, 32000),
    "4k": (4096, 11008, 4, 32000),
}
FP32_FMA_PER_SM_PER_CLOCK = 128          # float32 lanes of an SM: the scan's roofline is 2 * this * SMs * clock


def design_configs(width: int, ff: int, layers: int, vocab: int) -> tuple[dict, dict]:
    """A Zodosun configuration with heads of 128 and the Qwen2 configuration of the same width, depth, heads,
    feed-forward and vocabulary."""
    heads, kv = width // 128, max(1, width // 512)
    delta = {"type": "general_delta", "mixer": {"heads": heads, "dim": 128, "rank": 64},
             "mlp": {"kind": "dense", "ff": ff}}
    side = {"type": "parallel", "mlp": {"kind": "dense", "ff": ff}, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "bias_max": 4096,
                 "bias_rows": 64, "q_temp": {"coef": 0.1, "every": 256}},
        "right": {"heads": heads, "dim": 128, "vdim": 128,
                  "decay": [1.0 - 2.0 ** -(3 + 5 * h / max(1, heads - 1)) for h in range(heads)]}}}
    zod = {"architecture": "Zodosun", "vocab": vocab, "width": width, "logit_scale": 1.0,
           "norm": {"eps": 1e-6, "groups": 1}, "max_positions": 8192,
           "layers": [side if i % 4 == 2 else delta for i in range(layers)]}
    qwen = {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "hidden_act": "silu", "torch_dtype": "bfloat16",
            "num_hidden_layers": layers, "hidden_size": width, "num_attention_heads": heads, "num_key_value_heads": kv,
            "head_dim": 128, "intermediate_size": ff, "vocab_size": vocab, "rope_theta": 1e6, "rms_norm_eps": 1e-6,
            "tie_word_embeddings": False, "use_sliding_window": False, "sliding_window": None,
            "max_window_layers": layers, "max_position_embeddings": 8192}
    return zod, qwen


def rirudra_config(width: int, ff: int, layers: int, vocab: int) -> dict:
    """A Rirudra configuration of the given width: attention through a latent of 96 values and a rotated part of 32
    (heads of 96 + 32 key and 128 value entries), a state-space layer with twice the width inside (heads of 64, a
    state of 128), a gated delta rule with heads of 128 on half as many key heads; layers in that order, every
    fourth again attention."""
    heads = width // 128
    mlp = {"kind": "dense", "ff": ff}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": 96, "rot_dim": 32, "vdim": 128, "q_rank": 3 * width // 8, "kv_rank": 96,
        "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 32}}}
    ssm = {"type": "mamba2", "mlp": mlp, "mixer": {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1,
                                                    "norm_groups": 1, "conv": 4}}
    delta = {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128,
                                                    "vdim": 128, "conv": 4}}
    order = [latent, ssm, delta, latent]
    return {"architecture": "Rirudra", "vocab": vocab, "width": width, "embedding": {"scale": 8.0},
            "residual_mult": 0.5, "norm": {"eps": 1e-6}, "max_positions": 8192,
            "layers": [order[i % 4] for i in range(layers)]}


PAVISUN_WINDOW, PAVISUN_KEPT, PAVISUN_EXPERTS, PAVISUN_TOP, PAVISUN_STREAMS = 1024, 4, 8, 2, 4


def pavisun_config(width: int, ff: int, layers: int, vocab: int) -> dict:
    """A Pavisun configuration of the given width: heads of 128 on a quarter as many key heads; layers alternate
    between the mixer of unit-size q and k (distance slopes, a window of 1,024 that keeps the first 4 tokens, an
    output gate) and the rotating mixer whose values are its keys (capped scores, a window of 1,024, rotation
    stretched 8 times); 8 experts of half the feed-forward width of which a token uses 2 (as many products per
    token as the dense feed-forward has); 4 residual streams; capped logits."""
    heads, kv = width // 128, max(1, width // 512)
    mlp = {"kind": "moe", "expert": {"ff": ff // PAVISUN_TOP}, "router": {"experts": PAVISUN_EXPERTS, "top": PAVISUN_TOP}}
    unit = {"type": "attention_2", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 1.0,
        "mask": {"size": PAVISUN_WINDOW, "keep_first": PAVISUN_KEPT}}}
    rot = {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
        "mask": {"size": PAVISUN_WINDOW},
        "rot": {"base": 1e6, "dims": 128, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    return {"architecture": "Pavisun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "streams": PAVISUN_STREAMS, "logit_softcap": 30.0, "max_positions": 8192,
            "layers": [unit if i % 2 == 0 else rot for i in range(layers)]}


FURESUN_WINDOW, FURESUN_EXPERTS, FURESUN_TOP = 1024, 8, 2


def furesun_config(width: int, ff: int, layers: int, vocab: int) -> dict:
    """A Furesun configuration of the given width, heads of 128: attention through a latent of 96 values and a
    rotated part of 32 (rotation stretched 8 times, a window of 1,024) with a dense gelu feed-forward; a matrix
    memory with heads of 128 x 128; softmax attention on a quarter as many key heads (whole-row q/k norm, capped
    scores, a window of 1,024, a sink); the same attention reading the third layer's keys; the last three layers
    with 8 experts of a quarter of the feed-forward width of which a token uses 2, and a shared expert of half of it
    (as many products per token as the dense feed-forward has); capped logits."""
    heads, kv = width // 128, max(1, width // 512)
    moe = {"kind": "moe", "expert": {"ff": ff // 4}, "shared": {"ff": ff // 2},
           "router": {"experts": FURESUN_EXPERTS, "top": FURESUN_TOP, "scale": 2.0}}
    latent = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff}, "mixer": {
        "heads": heads, "dim": 96, "rot_dim": 32, "vdim": 128, "kv_rank": 96, "scale": 128 ** -0.5,
        "mask": {"size": FURESUN_WINDOW},
        "rot": {"base": 1e4, "dims": 32, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    memory = {"type": "mlstm", "mlp": moe, "mixer": {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    attn = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
            "mask": {"size": FURESUN_WINDOW}, "rot": {"base": 1e6, "dims": 64}}
    order = [latent, memory, {"type": "attention", "mlp": moe, "mixer": attn},
             {"type": "attention", "mlp": moe, "mixer": {**attn, "kv_from": 2}}]
    return {"architecture": "Furesun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "max_positions": 8192, "layers": [order[i] for i in range(min(layers, 4))]}


GOKAPEL_CHUNK, GOKAPEL_EXPERTS, GOKAPEL_TOP, GOKAPEL_STREAMS, GOKAPEL_RANK = 1100, 8, 2, 2, 128


def gokapel_config(width: int, ff: int, layers: int, vocab: int) -> dict:
    """A Gokapel configuration of the given width, heads of 128: the delta rule with a decay per key channel (half as
    many key heads, two-step projections of inner width 128); attention in chunks of 1,100 (a decoded token after 2,048 then sees about a thousand keys) on a quarter as many key
    heads beside a minGRU as wide as the model; feed-forwards without a gate, half again as wide as the gated ones of
    the other decoders (as many weights), dense in the first and last layer, in the second and third as 8 experts of a
    quarter of that in 4 groups, of which a token uses 2 of 2 groups, and a shared one of half; 2 residual streams."""
    heads, kv = width // 128, max(1, width // 512)
    f = 3 * ff // 2
    plain = {"kind": "dense", "ff": f}
    moe = {"kind": "moe", "expert": {"ff": f // 4}, "shared": {"ff": f // 2},
           "router": {"experts": GOKAPEL_EXPERTS, "top": GOKAPEL_TOP, "groups": {"count": 4, "keep": 2}}}
    delta = {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "conv": 4,
             "decay_rank": GOKAPEL_RANK, "gate_rank": GOKAPEL_RANK}
    side = {"left": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "mask": {"size": GOKAPEL_CHUNK}, "rot": {"base": 1e6, "dims": 64}},
            "left_scale": 0.7, "right": {"width": width}, "right_scale": 0.7}
    order = [("channel_delta", delta, plain), ("parallel", side, moe), ("channel_delta", delta, moe), ("parallel", side, plain)]
    return {"architecture": "Gokapel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "streams": GOKAPEL_STREAMS,
            "residual_mult": 0.7, "embedding": {"scale": 8.0}, "max_positions": 8192,
            "layers": [{"type": t, "mixer": m, "mlp": l} for t, m, l in (order[i % 4] for i in range(layers))]}


def gokapel_roofline(rec: dict, pk: dict, P: int, sms: int) -> dict:
    """What the classes of the Gokapel decoder reach of their rooflines, beside the like classes of the Rirudra decoder
    (scan, convolution), of the Pavisun decoder (streams, experts) and of the Qwen2 decoder (attention, products)."""
    width, ff, layers = rec["width"], rec["ff"], rec["layers"]
    heads, kv, d = width // 128, max(1, width // 512), 128
    g, r, p, q = rec["gokapel"], rec["rirudra"], rec["pavisun"], rec["qwen2"]
    f, n_delta = 3 * ff // 2, 2
    fp32_tflops = 2 * FP32_FMA_PER_SM_PER_CLOCK * sms * 1900.0 * 1e6 / 1e12
    roof = {"fp32_fma_tflops_nominal": round(fp32_tflops, 1)}

    def us(model, when, names):
        return sum(model[when].get(k, 0.0) for k in names) * 1e-6

    def tensor(name, flops, model, when, names):
        roof[name + ".frac_of_bf16"] = round(flops / us(model, when, names) / 1e12 / pk["bf16_tflops"], 3)

    def hbm(name, nbytes, model, when, names):
        roof[name + ".frac_of_hbm"] = round(nbytes / us(model, when, names) / 1e9 / pk["hbm_gbs"], 3)

    pre, dec = "prefill_classes_us", "decode_b64_classes_us"
    C = GOKAPEL_CHUNK
    tensor("gokapel.prefill.attention", 4 * heads * d * sum(i % C + 1 for i in range(P)) * 2, g, pre, ["attention"])
    tensor("qwen2.prefill.attention", 4 * heads * d * P * (P + 1) / 2 * layers, q, pre, ["attention"])
    seen = sum(min(i + 1, PAVISUN_WINDOW) for i in range(P))
    tensor("pavisun.prefill.attention", 4 * heads * d * seen * layers, p, pre, ["attention"])
    # delta rules: per token and head 8 d e operations; the state-space layer of the Rirudra decoder 5 d e
    delta_state, ssm_state = heads * 128 * 128, (2 * width // 64) * 128 * 64
    roof["gokapel.prefill.scan.frac_of_fp32_fma"] = round(P * 8 * delta_state * n_delta / us(g, pre, ["scan"]) / 1e12 / fp32_tflops, 3)
    roof["rirudra.prefill.scan.frac_of_fp32_fma"] = round(
        P * (5 * ssm_state + 8 * delta_state) / us(r, pre, ["scan"]) / 1e12 / fp32_tflops, 3)
    hbm("gokapel.decode_b64.scan", 64 * delta_state * 4 * 2 * n_delta, g, dec, ["scan"])
    hbm("rirudra.decode_b64.scan", 64 * (ssm_state + delta_state) * 4 * 2, r, dec, ["scan"])
    # convolutions: float32 channels read and written once
    ch_g, ch_r = 2 * max(1, heads // 2) * 128 + heads * 128, (2 * width + 256) + 2 * max(1, heads // 2) * 128 + heads * 128
    hbm("gokapel.prefill.conv", P * 8 * ch_g * n_delta, g, pre, ["conv"])
    hbm("rirudra.prefill.conv", P * 8 * ch_r, r, pre, ["conv"])
    # the minGRU: three float32 columns read, a bfloat16 one written; the two-step projections: two float32 results
    # written, one read and written once more
    hbm("gokapel.prefill.gru", P * width * (3 * 4 + 2) * 2, g, pre, ["gru"])
    hbm("gokapel.prefill.decay", P * heads * 128 * (4 + 4 + 8) * n_delta, g, pre, ["decay"])
    # between the sublayers: streams read and written, the sublayer's float32 result (and here its gate) read, a rounded
    # norm written
    S = GOKAPEL_STREAMS
    hbm("gokapel.prefill.between_sublayers", P * width * (8 * S + 4 + 4 + 2) * 2 * layers, g, pre, ["norms"])
    S = PAVISUN_STREAMS
    hbm("pavisun.prefill.between_sublayers", P * width * (8 * S + 4 + 2) * 2 * layers, p, pre, ["norms"])
    # products: everything that reads a mixer's input, and the output products
    n_in = [2 * max(1, heads // 2) * 128 + heads * 128 + width + 2 * GOKAPEL_RANK + heads, (heads + 2 * kv) * 128 + 4 * width]
    tensor("gokapel.prefill.qkv", 2 * P * width * sum(n_in) * 2, g, pre, ["qkv"])
    tensor("qwen2.prefill.qkv", 2 * P * width * (heads + 2 * kv) * 128 * layers, q, pre, ["qkv"])
    tensor("gokapel.prefill.o", 2 * P * width * (heads * 128 * 4 + 2 * width), g, pre, ["o"])
    tensor("qwen2.prefill.o", 2 * P * width * heads * 128 * layers, q, pre, ["o"])
    tensor("gokapel.prefill.dense_feed_forward", 4 * P * width * f * 2, g, pre, ["up", "down"])
    tensor("qwen2.prefill.dense_feed_forward", 6 * P * width * ff * layers, q, pre, ["gate_up", "down"])
    tensor("gokapel.prefill.experts", 4 * P * width * (f // 4) * GOKAPEL_TOP * 2, g, pre, ["experts"])
    tensor("pavisun.prefill.experts", 6 * P * width * (ff // PAVISUN_TOP) * PAVISUN_TOP * layers, p, pre, ["experts"])
    tensor("gokapel.prefill.shared_expert", 4 * P * width * (f // 2) * 2, g, pre, ["shared_expert"])
    tensor("gokapel.prefill.residual_gate_and_router", 2 * P * width * width * layers, g, pre, ["residual_gate", "router"])
    hbm("gokapel.decode_b64.attention", 64 * ((P + 16) % C + 1) * 2 * kv * d * 2 * 2, g, dec, ["attention"])
    hbm("qwen2.decode_b64.attention", 64 * (P + 16) * 2 * kv * d * 2 * layers, q, dec, ["attention"])
    hbm("gokapel.decode_b64.products", 2 * width * (sum(n_in) * 2 + heads * 128 * 4 + 2 * width), g, dec, ["qkv", "o"])
    hbm("qwen2.decode_b64.products", 2 * width * ((heads + 2 * kv) * 128 + heads * 128) * layers, q, dec, ["qkv", "o"])
    hbm("gokapel.decode_b64.dense_feed_forward", 2 * width * f * 2 * 2, g, dec, ["up", "down"])
    hbm("qwen2.decode_b64.dense_feed_forward", 3 * width * ff * 2 * layers, q, dec, ["gate_up", "down"])
    hbm("gokapel.decode_b64.experts", 2 * width * (f // 4) * GOKAPEL_EXPERTS * 2 * 2, g, dec, ["experts"])
    hbm("pavisun.decode_b64.experts", 3 * width * (ff // PAVISUN_TOP) * PAVISUN_EXPERTS * 2 * layers, p, dec, ["experts"])
    hbm("gokapel.decode_b64.shared_expert", 2 * width * (f // 2) * 2 * 2, g, dec, ["shared_expert"])
    hbm("gokapel.decode_b64.between_sublayers", 64 * width * (8 * GOKAPEL_STREAMS + 10) * 2 * layers, g, dec, ["norms"])
    hbm("pavisun.decode_b64.between_sublayers", 64 * width * (8 * PAVISUN_STREAMS + 6) * 2 * layers, p, dec, ["norms"])
    return roof


SAFURAX_WINDOW, SAFURAX_EXPERTS, SAFURAX_TOP = 1024, 8, 2


def safurax_config(width: int, ff: int, layers: int, vocab: int) -> dict:
    """A Safurax configuration of the given width: a difference of two maps of 64 over values of 128 on a quarter as many
    key/value heads, with a dense feed-forward; attention through a latent of 128 values without positions, queries
    through a latent of half the width; attention through a latent of 96 values and a rotated part of 32 (a window of
    1,024, a sink, a gate per head); the same reading the third layer's latents; the last three layers with 8 experts
    of a quarter of the feed-forward width of which a token uses 2, and a gated shared expert of half of it (as many
    products per token as the dense feed-forward has)."""
    heads, kv = width // 128, max(1, width // 512)
    moe = {"kind": "moe", "expert": {"ff": ff // 4}, "shared": {"ff": ff // 2},
           "router": {"experts": SAFURAX_EXPERTS, "top": SAFURAX_TOP}}
    maps = {"heads": heads, "kv_heads": kv, "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.4,
            "rot": {"base": 5e4, "dims": 64, "scaling": {"factor": 8.0}}}
    plain = {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": 128, "q_rank": width // 2, "scale": 128 ** -0.5}
    windowed = {"heads": heads, "dim": 96, "rot_dim": 32, "vdim": 128, "kv_rank": 96, "scale": 128 ** -0.5,
                "mask": {"size": SAFURAX_WINDOW}, "rot": {"base": 1e4, "dims": 32}}
    order = [("attention", maps, {"kind": "dense", "ff": ff}), ("latent_attention", plain, moe),
             ("latent_attention_2", windowed, moe), ("latent_attention_2", {**windowed, "kv_from": 2}, moe)]
    return {"architecture": "Safurax", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0},
            "max_positions": 8192, "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in order[:layers]]}


def safurax_roofline(rec: dict, pk: dict, P: int, sms: int) -> dict:
    """What the classes of the Safurax decoder reach of their rooflines, beside the like classes of the Furesun decoder
    (latent attention, experts) and of the Qwen2 decoder (attention, products, norms)."""
    width, ff, layers = rec["width"], rec["ff"], rec["layers"]
    heads, kv, d = width // 128, max(1, width // 512), 128
    s, f, q = rec["safurax"], rec["furesun"], rec["qwen2"]
    roof: dict = {}

    def us(model, when, names):
        return sum(model[when].get(k, 0.0) for k in names) * 1e-6

    def tensor(name, flops, model, when, names):
        roof[name + ".frac_of_bf16"] = round(flops / us(model, when, names) / 1e12 / pk["bf16_tflops"], 3)

    def hbm(name, nbytes, model, when, names):
        roof[name + ".frac_of_hbm"] = round(nbytes / us(model, when, names) / 1e9 / pk["hbm_gbs"], 3)

    pre, dec = "prefill_classes_us", "decode_b64_classes_us"
    pairs, Wd, E = P * (P + 1) / 2, SAFURAX_WINDOW, SAFURAX_EXPERTS
    seen = sum(min(i + 1, Wd) for i in range(P))
    # the maps' scores (two of 64 entries) and their sums of values (two of 128), the plain latent and two windowed ones
    tensor("safurax.prefill.attention", heads * ((4 * 64 + 4 * d) * pairs + 4 * d * (pairs + 2 * seen)), s, pre, ["attention"])
    tensor("furesun.prefill.attention", 4 * heads * d * seen * 3, f, pre, ["attention"])
    tensor("qwen2.prefill.attention", 4 * heads * d * pairs * layers, q, pre, ["attention"])
    # two float32 results per head in, one rounded row out
    hbm("safurax.prefill.difference", P * heads * d * (2 * 4 + 2), s, pre, ["difference"])
    # encodings.  Maps: the float32 projections read, two widened queries per head, keys and values (rows and pages)
    # written.  Latents: float32 projections read, rounded ones written; the windowed layers' heads (q, k, v float32 in,
    # bfloat16 out) and their gated, narrowed results
    maps = (heads + 2 * kv) * d * 4 + 2 * heads * d * 2 + 2 * 2 * kv * d * 2
    lat1 = (width // 2 + 128) * (4 + 2) + 128 * 2
    lat2 = heads * (128 + 96 + 128) * 4 + 3 * heads * d * 2
    hbm("safurax.prefill.encodings", P * (maps + lat1 + 2 * lat2 + 128 * (4 + 2 + 2)), s, pre, ["rotary"])
    f_attn = (heads + 2 * kv) * d * 4 + (heads + 4 * kv) * d * 2 + heads * d * (4 + 2)
    hbm("furesun.prefill.encodings", P * (f_attn + lat2 + 128 * (4 + 2 + 2) + heads * d * 4), f, pre, ["rotary"])
    n_in = [(heads + 2 * kv) * d + heads, width // 2 + 128, heads * d + 128 + heads, heads * d + heads]
    up1, up2 = width // 2 * heads * d + 2 * 128 * heads * d, 96 * heads * (96 + 128)
    tensor("safurax.prefill.qkv", 2 * P * (width * sum(n_in) + up1 + 2 * up2), s, pre, ["qkv"])
    tensor("qwen2.prefill.qkv", 2 * P * width * (heads + 2 * kv) * d * layers, q, pre, ["qkv"])
    tensor("safurax.prefill.o", 2 * P * width * heads * d * 4, s, pre, ["o"])
    tensor("qwen2.prefill.o", 2 * P * width * heads * d * layers, q, pre, ["o"])
    ff_flops = 6 * P * width * ff
    tensor("safurax.prefill.dense_feed_forward", ff_flops, s, pre, ["gate_up", "down"])
    tensor("furesun.prefill.dense_feed_forward", ff_flops, f, pre, ["gate_up", "down"])
    tensor("qwen2.prefill.dense_feed_forward", ff_flops * layers, q, pre, ["gate_up", "down"])
    tensor("safurax.prefill.experts", ff_flops * 3 / 2, s, pre, ["experts", "router"])
    tensor("furesun.prefill.experts", ff_flops * 3 / 2, f, pre, ["experts"])
    tensor("safurax.prefill.shared_expert", ff_flops * 3 / 2, s, pre, ["shared_expert"])
    tensor("furesun.prefill.shared_expert", ff_flops * 3 / 2, f, pre, ["shared_expert"])
    hbm("safurax.prefill.norms", P * width * (4 + 2) * 2 * 4, s, pre, ["norms"])
    hbm("qwen2.prefill.norms", P * width * (4 + 2) * 2 * layers, q, pre, ["norms"])
    n = P + 16
    row = 2 * kv * d * 2
    hbm("safurax.decode_b64.attention", 64 * (n * row + n * 128 * 2 + 2 * min(n, Wd) * 128 * 2), s, dec, ["attention"])
    hbm("furesun.decode_b64.attention", 64 * min(n, Wd) * (128 * 2 + 2 * row), f, dec, ["attention"])
    hbm("qwen2.decode_b64.attention", 64 * n * row * layers, q, dec, ["attention"])
    # decode: the latents' per-head matrices read once (they ride in this class), float32 projections and rounded rows
    up = 2 * heads * d * (2 * 128 + 2 * 2 * 96)
    act = 64 * heads * 3 * (4 * 128 + 2 * 128 * 3)
    hbm("safurax.decode_b64.encodings", up + act + 64 * maps, s, dec, ["rotary"])
    hbm("furesun.decode_b64.encodings", 2 * heads * d * 2 * 96 + act // 3 + 64 * f_attn, f, dec, ["rotary"])
    hbm("safurax.decode_b64.products", 2 * (width * (sum(n_in) + 4 * heads * d) + width // 2 * heads * d), s, dec, ["qkv", "o"])
    hbm("qwen2.decode_b64.products", 2 * width * ((heads + 2 * kv) * d + heads * d) * layers, q, dec, ["qkv", "o"])
    hbm("safurax.decode_b64.dense_feed_forward", 3 * width * ff * 2, s, dec, ["gate_up", "down"])
    hbm("furesun.decode_b64.dense_feed_forward", 3 * width * ff * 2, f, dec, ["gate_up", "down"])
    hbm("qwen2.decode_b64.dense_feed_forward", 3 * width * ff * 2 * layers, q, dec, ["gate_up", "down"])
    hbm("safurax.decode_b64.experts", 3 * width * (ff // 4) * E * 2 * 3, s, dec, ["experts", "router"])
    hbm("furesun.decode_b64.experts", 3 * width * (ff // 4) * E * 2 * 3, f, dec, ["experts"])
    hbm("safurax.decode_b64.shared_expert", 3 * width * (ff // 2) * 2 * 3, s, dec, ["shared_expert"])
    hbm("furesun.decode_b64.shared_expert", 3 * width * (ff // 2) * 2 * 3, f, dec, ["shared_expert"])
    hbm("safurax.decode_b64.norms", 64 * width * (4 + 2) * 2 * 4, s, dec, ["norms"])
    hbm("qwen2.decode_b64.norms", 64 * width * (4 + 2) * 2 * layers, q, dec, ["norms"])
    return roof


def furesun_roofline(rec: dict, pk: dict, P: int, sms: int) -> dict:
    """What the classes of the Furesun decoder reach of their rooflines, beside the like classes of the Qwen2
    decoder (attention, feed-forward, the kernels between the sublayers) and of the Rirudra decoder (the scan)."""
    width, ff, layers = rec["width"], rec["ff"], rec["layers"]
    heads, kv, d = width // 128, max(1, width // 512), 128
    f, q, r = rec["furesun"], rec["qwen2"], rec["rirudra"]
    Wd, E, top = FURESUN_WINDOW, FURESUN_EXPERTS, FURESUN_TOP
    fp32_tflops = 2 * FP32_FMA_PER_SM_PER_CLOCK * sms * 1900.0 * 1e6 / 1e12

    def frac_tensor(flops, us):
        return round(flops / (us * 1e-6) / 1e12 / pk["bf16_tflops"], 3)

    def frac_hbm(nbytes, us):
        return round(nbytes / (us * 1e-6) / 1e9 / pk["hbm_gbs"], 3)

    seen = sum(min(i + 1, Wd) for i in range(P))                        # keys a prompt's rows see in a window
    roof = {"fp32_fma_tflops_nominal": round(fp32_tflops, 1)}
    roof["furesun.prefill.attention.frac_of_bf16"] = frac_tensor(4 * heads * d * seen * 3, f["prefill_classes_us"]["attention"])
    roof["qwen2.prefill.attention.frac_of_bf16"] = frac_tensor(
        4 * heads * d * P * (P + 1) / 2 * layers, q["prefill_classes_us"]["attention"])
    # the memory: per token and head 2 d e' multiply-adds for the update and 2 d e' for the read, e' = 132 columns
    state = heads * 128 * 132
    roof["furesun.prefill.scan.frac_of_fp32_fma"] = round(
        P * 5 * state / (f["prefill_classes_us"]["scan"] * 1e-6) / 1e12 / fp32_tflops, 3)
    ssm_state, delta_state = (2 * width // 64) * 128 * 64, heads * 128 * 128
    roof["rirudra.prefill.scan.frac_of_fp32_fma"] = round(
        P * (5 * ssm_state + 8 * delta_state) / (r["prefill_classes_us"]["scan"] * 1e-6) / 1e12 / fp32_tflops, 3)
    roof["furesun.decode_b64.scan.frac_of_hbm"] = frac_hbm(64 * state * 4 * 2, f["decode_b64_classes_us"]["scan"])
    roof["rirudra.decode_b64.scan.frac_of_hbm"] = frac_hbm(
        64 * (ssm_state + delta_state) * 4 * 2, r["decode_b64_classes_us"]["scan"])
    # the feed-forwards of a prompt: one dense layer and three of experts (2 of 8 small ones and the shared one)
    ff_flops = 6 * P * width * ff
    roof["furesun.prefill.feed_forward.frac_of_bf16"] = frac_tensor(
        ff_flops * 4, sum(f["prefill_classes_us"].get(k, 0.0) for k in ("gate_up", "down", "experts", "shared_expert")))
    roof["qwen2.prefill.feed_forward.frac_of_bf16"] = frac_tensor(
        ff_flops * layers, q["prefill_classes_us"]["gate_up"] + q["prefill_classes_us"]["down"])
    # between the sublayers: the sublayer's float32 result read, the stream read and written, a rounded copy written;
    # the plain decoder reads the stream and writes a rounded norm (its sum rides in a product's last step)
    roof["furesun.prefill.between_sublayers.frac_of_hbm"] = frac_hbm(
        P * width * (4 + 4 + 4 + 2) * 2 * 4, f["prefill_classes_us"]["norms"])
    roof["qwen2.prefill.between_sublayers.frac_of_hbm"] = frac_hbm(
        P * width * (4 + 2) * 2 * layers, q["prefill_classes_us"]["norms"])
    keys = min(P + 16, Wd)
    roof["furesun.decode_b64.attention.frac_of_hbm"] = frac_hbm(
        64 * keys * (128 * 2 + 2 * 2 * kv * d * 2), f["decode_b64_classes_us"]["attention"])
    roof["qwen2.decode_b64.attention.frac_of_hbm"] = frac_hbm(
        64 * (P + 16) * 2 * kv * d * 2 * layers, q["decode_b64_classes_us"]["attention"])
    roof["furesun.decode_b64.feed_forward.frac_of_hbm"] = frac_hbm(
        3 * width * 2 * (ff + 3 * (E * (ff // 4) + ff // 2)),
        sum(f["decode_b64_classes_us"].get(k, 0.0) for k in ("gate_up", "down", "experts", "shared_expert")))
    roof["qwen2.decode_b64.feed_forward.frac_of_hbm"] = frac_hbm(
        3 * width * ff * 2 * layers, q["decode_b64_classes_us"]["gate_up"] + q["decode_b64_classes_us"]["down"])
    return roof


def pavisun_roofline(rec: dict, pk: dict, P: int) -> dict:
    """What the classes of the Pavisun decoder reach of their rooflines, beside the like classes of the Qwen2
    decoder: attention (tensor throughput in a prompt, key and value bytes in decoding), the feed-forward (tensor
    throughput in a prompt, weight bytes in decoding) and the kernels between the sublayers (bytes)."""
    width, ff, layers = rec["width"], rec["ff"], rec["layers"]
    heads, kv, d = width // 128, max(1, width // 512), 128
    p, q = rec["pavisun"], rec["qwen2"]
    n_unit = (layers + 1) // 2
    n_rot = layers - n_unit
    Wd, K, S, E, top = PAVISUN_WINDOW, PAVISUN_KEPT, PAVISUN_STREAMS, PAVISUN_EXPERTS, PAVISUN_TOP

    def frac_tensor(flops, us):
        return round(flops / (us * 1e-6) / 1e12 / pk["bf16_tflops"], 3)

    def frac_hbm(nbytes, us):
        return round(nbytes / (us * 1e-6) / 1e9 / pk["hbm_gbs"], 3)

    seen_win = sum(min(i + 1, Wd) for i in range(P))                    # keys a prompt's rows see in a window
    seen_kept = seen_win + sum(min(K, max(0, i + 1 - Wd)) for i in range(P))
    roof = {}
    roof["pavisun.prefill.attention.frac_of_bf16"] = frac_tensor(
        4 * heads * d * (seen_kept * n_unit + seen_win * n_rot), p["prefill_classes_us"]["attention"])
    roof["qwen2.prefill.attention.frac_of_bf16"] = frac_tensor(
        4 * heads * d * P * (P + 1) / 2 * layers, q["prefill_classes_us"]["attention"])
    n_ff = layers
    roof["pavisun.prefill.experts.frac_of_bf16"] = frac_tensor(
        6 * P * top * width * (ff // top) * n_ff, p["prefill_classes_us"]["experts"])
    roof["qwen2.prefill.feed_forward.frac_of_bf16"] = frac_tensor(
        6 * P * width * ff * layers, q["prefill_classes_us"]["gate_up"] + q["prefill_classes_us"]["down"])
    # between the sublayers: the streams are read and written once per sublayer (float32), the normed sum written
    # (bfloat16) and the sublayer's result read (float32); the plain decoder reads and writes one residual row
    between_p = P * width * (2 * S * 4 + 2 + 4) * 2 * layers
    between_q = P * width * (2 * 2 + 2 + 2) * 2 * layers
    roof["pavisun.prefill.between_sublayers.frac_of_hbm"] = frac_hbm(between_p, p["prefill_classes_us"]["norms"])
    roof["qwen2.prefill.between_sublayers.frac_of_hbm"] = frac_hbm(between_q, q["prefill_classes_us"]["norms"])
    # decoding, 64 sequences that hold P + 16 tokens: the window's keys and values (the rotating mixer's values are
    # its keys before the rotation: rows of their own in the cache), and the kept first tokens
    keys = min(P + 16, Wd)
    row = kv * d * 2
    roof["pavisun.decode_b64.attention.frac_of_hbm"] = frac_hbm(
        64 * ((keys + K) * 2 * row * n_unit + keys * 2 * row * n_rot), p["decode_b64_classes_us"]["attention"])
    roof["qwen2.decode_b64.attention.frac_of_hbm"] = frac_hbm(
        64 * (P + 16) * 2 * row * layers, q["decode_b64_classes_us"]["attention"])
    roof["pavisun.decode_b64.experts.frac_of_hbm"] = frac_hbm(
        E * 3 * width * (ff // top) * 2 * n_ff, p["decode_b64_classes_us"]["experts"])
    roof["qwen2.decode_b64.feed_forward.frac_of_hbm"] = frac_hbm(
        3 * width * ff * 2 * layers, q["decode_b64_classes_us"]["gate_up"] + q["decode_b64_classes_us"]["down"])
    return roof


def rirudra_roofline(rec: dict, pk: dict, P: int, sms: int) -> dict:
    """What the attention and scan classes of the Rirudra decoder reach of their rooflines, beside the like classes
    of the Qwen2 decoder (attention) and of the Zodosun decoder (scans)."""
    width, layers = rec["width"], rec["layers"]
    heads = width // 128
    r, q, z = rec["rirudra"], rec["qwen2"], rec["zodosun"]
    kinds = [("latent", "ssm", "delta", "latent")[i % 4] for i in range(layers)]
    n_lat, n_ssm, n_delta = kinds.count("latent"), kinds.count("ssm"), kinds.count("delta")
    fp32_tflops = 2 * FP32_FMA_PER_SM_PER_CLOCK * sms * 1900.0 * 1e6 / 1e12
    roof = {"fp32_fma_tflops_nominal": round(fp32_tflops, 1)}
    attn_flops = 4 * heads * 128 * P * (P + 1) / 2                      # per layer, heads of 128 either way
    roof["rirudra.prefill.attention.frac_of_bf16"] = round(
        attn_flops * n_lat / (r["prefill_classes_us"]["attention"] * 1e-6) / 1e12 / pk["bf16_tflops"], 3)
    roof["qwen2.prefill.attention.frac_of_bf16"] = round(
        attn_flops * layers / (q["prefill_classes_us"]["attention"] * 1e-6) / 1e12 / pk["bf16_tflops"], 3)
    ssm_state, delta_state = (2 * width // 64) * 128 * 64, heads * 128 * 128          # floats per sequence and layer
    scan_flops = P * (5 * ssm_state * n_ssm + 8 * delta_state * n_delta)
    roof["rirudra.prefill.scan.frac_of_fp32_fma"] = round(
        scan_flops / (r["prefill_classes_us"]["scan"] * 1e-6) / 1e12 / fp32_tflops, 3)
    z_delta = sum(1 for i in range(layers) if i % 4 != 2)
    roof["zodosun.prefill.scan.frac_of_fp32_fma"] = round(
        P * heads * 128 * 128 * (8 * z_delta + 5 * (layers - z_delta)) / (z["prefill_classes_us"]["scan"] * 1e-6)
        / 1e12 / fp32_tflops, 3)
    roof["rirudra.decode_b64.scan.frac_of_hbm"] = round(
        64 * (ssm_state * n_ssm + delta_state * n_delta) * 4 * 2 / (r["decode_b64_classes_us"]["scan"] * 1e-6) / 1e9
        / pk["hbm_gbs"], 3)
    roof["zodosun.decode_b64.scan.frac_of_hbm"] = round(
        64 * heads * 128 * 128 * 4 * 2 * layers / (z["decode_b64_classes_us"]["scan"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
    kv_row = 2 * max(1, width // 512) * 128 * 2
    roof["rirudra.decode_b64.attention.frac_of_hbm"] = round(
        64 * (P + 16) * 128 * 2 * n_lat / (r["decode_b64_classes_us"]["attention"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
    roof["qwen2.decode_b64.attention.frac_of_hbm"] = round(
        64 * (P + 16) * kv_row * layers / (q["decode_b64_classes_us"]["attention"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
    return roof


def design_compare(args) -> int:
    """Prefill and decode of the named decoder and of the Qwen2 decoder of equal size, random weights, bfloat16:
    device time of a 2,048-token prompt, of decode steps at batch 8 and 64 (replayed graphs), and the time by
    class of kernel with what each class reaches of its roofline."""
    import torch
    import tq_kv_b200 as tq
    from tq_kv_b200 import kernels
    from tq_kv_b200.engine import StepRow
    pk, pk_src = peaks()
    gen = torch.Generator().manual_seed(0)
    sms = torch.cuda.get_device_properties(0).multi_processor_count
    P, ctx = args.prompt, args.prompt + 512
    out = {"design": args.design, "beside": "qwen2", "dtype": "bf16", "data": "synthetic (random weights)",
           "peaks": {**pk, "source": pk_src}, "prompt": P, "sizes": {}}
    with ClockSampler() as clocks:
        for name in args.sizes.split(","):
            width, ff, layers, vocab = DESIGN_SIZES[name]
            rec = out["sizes"][name] = {"width": width, "ff": ff, "layers": layers, "vocab": vocab}
            zod, qwen = design_configs(width, ff, layers, vocab)
            models = [("zodosun", zod), ("qwen2", qwen)]
            if args.design == "rirudra":
                models.insert(0, ("rirudra", rirudra_config(width, ff, layers, vocab)))
            if args.design == "pavisun":
                models = [("pavisun", pavisun_config(width, ff, layers, vocab)), ("qwen2", qwen)]
            if args.design == "furesun":
                models = [("furesun", furesun_config(width, ff, layers, vocab)),
                          ("rirudra", rirudra_config(width, ff, layers, vocab)), ("qwen2", qwen)]
            if args.design == "gokapel":
                models = [("gokapel", gokapel_config(width, ff, layers, vocab)),
                          ("rirudra", rirudra_config(width, ff, layers, vocab)),
                          ("pavisun", pavisun_config(width, ff, layers, vocab)), ("qwen2", qwen)]
            if args.design == "safurax":
                models = [("safurax", safurax_config(width, ff, layers, vocab)),
                          ("furesun", furesun_config(width, ff, layers, vocab)), ("qwen2", qwen)]
            for model, cfg in models:
                eng = tq.Engine.from_random(cfg, seed=0, dtype="bfloat16", max_slots=64, max_context=ctx,
                                            max_tokens=64 * ctx)
                r = rec[model] = {}

                def prompt_rows(n_rows):
                    slots = [eng.new_sequence() for _ in range(n_rows)]
                    return slots, [StepRow(s, torch.randint(0, vocab, (P,), generator=gen).tolist(), [P - 1]) for s in slots]

                # prefill: one prompt, device time after two warm-up runs
                times = []
                for i in range(2 + 5):
                    slots, rows = prompt_rows(1)
                    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                    torch.cuda.synchronize()
                    e0.record()
                    eng.step(rows)
                    e1.record()
                    torch.cuda.synchronize()
                    times.append(e0.elapsed_time(e1))
                    eng.release(slots[0])
                r["prefill_ms"] = round(statistics.median(times[2:]), 3)
                r["prefill_tok_s"] = round(P / (r["prefill_ms"] * 1e-3))

                def one_prompt():
                    slots, rows = prompt_rows(1)
                    eng.step(rows)
                    eng.release(slots[0])

                r["prefill_classes_us"] = {k: round(v, 1) for k, v in timed_by_class(one_prompt).items() if k != "start"}
                # decode: batches of 8 and 64 sequences that hold P tokens, replayed graphs, 64 timed steps
                for B in (8, 64):
                    slots = [eng.new_sequence() for _ in range(B)]
                    for a in range(0, B, 8):
                        eng.step([StepRow(s, torch.randint(0, vocab, (P,), generator=gen).tolist(), []) for s in slots[a:a + 8]])
                    toks = torch.randint(0, vocab, (16 + 64, B), generator=gen).tolist()
                    for i in range(16):
                        eng.step([StepRow(s, [toks[i][j]], [0]) for j, s in enumerate(slots)], keep_logits=False)
                    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                    torch.cuda.synchronize()
                    e0.record()
                    for i in range(16, 80):
                        eng.step([StepRow(s, [toks[i][j]], [0]) for j, s in enumerate(slots)], keep_logits=False)
                    e1.record()
                    torch.cuda.synchronize()
                    eng.check_status()
                    ms = e0.elapsed_time(e1) / 64
                    r[f"decode_b{B}_ms"] = round(ms, 4)
                    r[f"decode_b{B}_tok_s"] = round(B / (ms * 1e-3))
                    if B == 64:
                        eng.use_graphs = False

                        def one_step():
                            eng.step([StepRow(s, [(37 * j + 1) % vocab], [0]) for j, s in enumerate(slots)],
                                     keep_logits=False)

                        one_step()
                        r["decode_b64_classes_us"] = {k: round(v, 1) for k, v in timed_by_class(one_step).items()
                                                      if k != "start"}
                        eng.use_graphs = True
                    for s in slots:
                        eng.release(s)
                del eng
                torch.cuda.empty_cache()
            if args.design == "rirudra":
                rec["roofline"] = rirudra_roofline(rec, pk, P, sms)
                continue
            if args.design == "pavisun":
                rec["roofline"] = pavisun_roofline(rec, pk, P)
                continue
            if args.design == "furesun":
                rec["roofline"] = furesun_roofline(rec, pk, P, sms)
                continue
            if args.design == "gokapel":
                rec["roofline"] = gokapel_roofline(rec, pk, P, sms)
                continue
            if args.design == "safurax":
                rec["roofline"] = safurax_roofline(rec, pk, P, sms)
                continue
            # what the classes reach of their rooflines
            heads, d = width // 128, 128
            z, q = rec["zodosun"], rec["qwen2"]
            n_delta = sum(1 for i in range(layers) if i % 4 != 2)
            n_side = layers - n_delta
            mhz = 1900.0
            fp32_tflops = 2 * FP32_FMA_PER_SM_PER_CLOCK * sms * mhz * 1e6 / 1e12
            scan_flops = P * heads * d * d * (8 * n_delta + 5 * n_side)
            attn_flops = 4 * heads * d * P * (P + 1) / 2
            roof = rec["roofline"] = {"fp32_fma_tflops_nominal": round(fp32_tflops, 1)}
            roof["zodosun.prefill.scan.frac_of_fp32_fma"] = round(
                scan_flops / (z["prefill_classes_us"]["scan"] * 1e-6) / 1e12 / fp32_tflops, 3)
            roof["zodosun.prefill.attention.frac_of_bf16"] = round(
                attn_flops * n_side / (z["prefill_classes_us"]["attention"] * 1e-6) / 1e12 / pk["bf16_tflops"], 3)
            roof["qwen2.prefill.attention.frac_of_bf16"] = round(
                attn_flops * layers / (q["prefill_classes_us"]["attention"] * 1e-6) / 1e12 / pk["bf16_tflops"], 3)
            state_bytes = 64 * heads * d * d * 4 * 2 * layers            # every layer reads and writes a state per head
            kv_row = 2 * max(1, width // 512) * d * 2
            roof["zodosun.decode_b64.scan.frac_of_hbm"] = round(
                state_bytes / (z["decode_b64_classes_us"]["scan"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
            roof["zodosun.decode_b64.attention.frac_of_hbm"] = round(
                64 * (P + 16) * kv_row * n_side / (z["decode_b64_classes_us"]["attention"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
            roof["qwen2.decode_b64.attention.frac_of_hbm"] = round(
                64 * (P + 16) * kv_row * layers / (q["decode_b64_classes_us"]["attention"] * 1e-6) / 1e9 / pk["hbm_gbs"], 3)
    out["clocks"] = clocks.summary()
    out["gpu_launches"] = kernels.launches[0]
    print(json.dumps(out))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", default=None, choices=["zodosun", "rirudra", "pavisun", "furesun", "gokapel", "safurax"],
                    help="instead of the default workload: this design beside the Qwen2 decoder of equal size")
    ap.add_argument("--sizes", default="1k,2k,4k", help="with --design: which of the sizes 1k, 2k, 4k (the model's width)")
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=None, help="default 8 (64 with --workload unequal)")
    ap.add_argument("--shape", default="qwen2.5-7b")
    ap.add_argument("--workload", default="equal", choices=["equal", "unequal"],
                    help="equal: prompts of --prompt tokens; unequal: seeded lengths uniform in 64..4096, one prefill step")
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the shape has (named in config)")
    ap.add_argument("--context", type=int, default=None, help="default 4096 (8192 with --workload unequal)")
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--e2e-steps", type=int, default=128, help="the end-to-end run takes at least this many steps")
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 points and the prefill")
    ap.add_argument("--no-e2e", action="store_true", help="skip the end-to-end run (for profiler captures)")
    ap.add_argument("--no-kernels", action="store_true", help="skip the per-class kernel times")
    ap.add_argument("--prefill-only", action="store_true", help="time the 2,048-token prefill alone (profiler captures)")
    ap.add_argument("--no-graphs", action="store_true", help="launch decode kernels one by one (for profiler captures)")
    ap.add_argument("--gemm", default=None, choices=["tcgen05", "library"],
                    help="many-row bfloat16 products: this package's tcgen05 kernel or the library (default: the package's choice)")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference is a Rust workspace (no setup.py/pyproject.toml; pip: 'not installable') "
                          "and no cargo/rustc is installed"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.design is not None:
        return design_compare(args)
    if args.warmup < 3:
        args.warmup = 3
    unequal = args.workload == "unequal"
    if args.batch is None:
        args.batch = 64 if unequal else 8
    if args.context is None:
        args.context = 8192 if unequal else 4096

    import torch
    import tq_kv_b200 as tq
    from tq_kv_b200 import kernels
    from tq_kv_b200.engine import StepRow
    from tq_kv_b200.sampling import Sampler

    if args.gemm is not None:
        kernels.gemm.USE_TCGEN05 = args.gemm == "tcgen05"
    cfg = dict(tq.named_shape(args.shape))
    full_layers = cfg["num_hidden_layers"]
    n_layers = args.layers or full_layers
    cfg["num_hidden_layers"] = n_layers
    cfg["max_window_layers"] = n_layers
    V = cfg["vocab_size"]
    pk, pk_src = peaks()
    nums = model_numbers(cfg, n_layers)
    K, W = args.steps, args.warmup
    gen = torch.Generator().manual_seed(0)
    if unequal:
        lengths = torch.randint(64, 4097, (args.batch,), generator=gen).tolist()
        max_b = args.batch
        room = max(K + W, max(args.e2e_steps, K) + max(W, 48) + 1) + 2
        max_tokens = sum(-(-(n + room) // 64) * 64 for n in lengths)
    else:
        lengths = None
        max_b = args.batch if args.no_points else max(args.batch, 64)
        # the cache a full batch of full contexts needs, cut to what fits beside the weights where it must be
        max_tokens = max_b * args.context
        free = torch.cuda.mem_get_info()[0] - nums["weight_bytes"] - 2 * V * cfg["hidden_size"] - (12 << 30)
        fit = int(free // nums["kv_bytes_per_token"]) // 64 * 64
        max_tokens = max(64 * max_b, min(max_tokens, fit))
    # the timed steps sit in the middle of a run from `prompt` to `context` tokens
    span = args.context - args.prompt
    start_ctx = args.prompt + max(0, (span - K - W) // 2)
    if start_ctx + K + W > args.context:
        start_ctx = max(1, args.context - K - W)

    engine = tq.Engine.from_random(cfg, seed=0, dtype="bfloat16", max_slots=max_b, max_context=args.context,
                                   max_tokens=max_tokens)
    engine.use_graphs = not args.no_graphs
    dev = engine.runtime.device

    def fill(ctx_lens: list[int]) -> list[int]:
        """Slots holding that many random tokens each, prefilled a few rows at a time."""
        slots = [engine.new_sequence() for _ in ctx_lens]
        for a in range(0, len(slots), 4):
            rows = [StepRow(s, torch.randint(0, V, (n,), generator=gen).tolist(), [])
                    for s, n in zip(slots[a:a + 4], ctx_lens[a:a + 4])]
            engine.step(rows)
        return slots

    def decode_run(ctx_lens: list[int], steps: int, warmup: int):
        """Device time of `steps` decode steps launched back to back."""
        batch = len(ctx_lens)
        slots = fill(ctx_lens)
        sampler = Sampler(tq.GenerationParams.greedy(1), batch, V, dev)
        toks = torch.randint(0, V, (steps + warmup, batch), generator=gen).tolist()

        def one(i):
            logits = engine.step([StepRow(s, [toks[i][r]], [0]) for r, s in enumerate(slots)], keep_logits=False)
            kernels.sample(logits, sampler.out)

        for i in range(warmup):
            one(i)
        torch.cuda.synchronize()
        n0 = kernels.launches[0]
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for i in range(warmup, warmup + steps):
            one(i)
        e1.record()
        torch.cuda.synchronize()
        engine.check_status()
        ms = e0.elapsed_time(e1)
        launches = kernels.launches[0] - n0
        for s in slots:
            engine.release(s)
        return ms, launches

    e2e_warmup = max(W, 48)

    def e2e_run(prompts: list[list[int]], steps: int):
        """Tokens per second through Engine.generate(): host token ids in, every step's ids back on the host.
        As in the device-timed run, the first steps after the prompts are warm-up and are not timed (right
        after prompts of thousands of tokens the first dozen or two of decode steps run at the lower clocks
        that the prompts' matrix products left behind: 4.2 instead of 3.2 ms at batch 8); then `steps` steps are timed between the arrivals of their
        tokens on the host."""
        stamps: list[float] = []
        B = len(prompts)

        def on_token(i, t):
            stamps.append(time.perf_counter())             # the token is on the host now

        h2d0, stats = engine.h2d_bytes, {}
        engine.generate(prompts, tq.GenerationParams.greedy(e2e_warmup + steps + 1, stop_token_ids=()),
                        on_token=on_token, stats=stats)
        # every request yields the same number of tokens, a round of the batch at a time: the clock starts with
        # the last token of the last warm-up round
        first = e2e_warmup * B - 1
        n_timed = len(stamps) - 1 - first
        value = n_timed / (stamps[-1] - stamps[first])
        rounds = len(stamps) / B
        h2d = (engine.h2d_bytes - h2d0 + stats.get("h2d_bytes", 0)) / rounds
        return value, int(h2d), int(stats.get("d2h_bytes", 0) / rounds), n_timed // B

    def e2e_prompt(steps: int) -> int:
        """Prompt length at which `steps` generated tokens see the same mean context as the device-timed steps."""
        want = start_ctx + W + K / 2 - steps / 2 - e2e_warmup
        return int(max(args.prompt, min(want, args.context - steps - e2e_warmup - 2)))

    def prefill_run(prompt_lens: list[int]):
        """One step over prompts of these lengths, logits at each prompt's last place; after one warm-up."""
        ms = 0.0
        for _ in range(2):
            slots = [engine.new_sequence() for _ in prompt_lens]
            rows = [StepRow(s, torch.randint(0, V, (n,), generator=gen).tolist(), [n - 1])
                    for s, n in zip(slots, prompt_lens)]
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            engine.step(rows)
            e1.record()
            torch.cuda.synchronize()
            ms = e0.elapsed_time(e1)
            for s in slots:
                engine.release(s)
        T = sum(prompt_lens)
        attn = nums["attn_flops_per_key"] * sum(n * (n + 1) / 2 for n in prompt_lens)
        flops = 2 * T * n_layers * nums["layer_mm"] + attn + 2 * len(prompt_lens) * nums["head_mm"]
        return ms, T, flops, attn

    if args.prefill_only:
        ms, T, _, _ = prefill_run([args.prompt])
        print(json.dumps({"prefill_ms": round(ms, 3), "tokens": T, "layers": n_layers}))
        return 0

    ctx_lens = [n + 1 for n in lengths] if unequal else [start_ctx] * args.batch
    with ClockSampler() as clocks:
        ms, launches = decode_run(ctx_lens, K, W)
    ms_step = ms / K
    value = args.batch * K / (ms / 1e3)
    mean_cached = sum(ctx_lens) + args.batch * (W + K / 2)          # tokens in the cache, mean over the timed steps
    step_bytes = nums["weight_bytes"] + mean_cached * nums["kv_bytes_per_token"]
    achieved = step_bytes / (ms_step / 1e3) / 1e9

    rec = {
        "metric": f"decode tok/s ({args.shape} shape, bf16 random weights)", "value": round(value, 1),
        "unit": "tok/s", "n_gpus": 1, "steps": K, "warmup": W, "ms_per_step": round(ms_step, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "impl": "ours", "gpu_launches": launches,
        "config": {"model": args.shape, "layers": n_layers, "layers_full": full_layers,
                   "hidden_size": cfg["hidden_size"], "heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate_size": cfg["intermediate_size"], "vocab_size": V, "global_batch": args.batch,
                   "seq_len": args.context,
                   "prompt_len": "uniform 64..4096, seed 0" if unequal else args.prompt,
                   "decode_ctx_start": round(sum(ctx_lens) / args.batch) + W,
                   "cache_tokens": engine.cache.groups[0].book.n_pages * 64,
                   "parallelism": "single GPU", "weights": "random N(0,0.02) bf16",
                   "l2": f"a step reads {step_bytes / 1e9:.1f} GB of weights and cache, more than the 126 MB L2",
                   "peaks": pk_src},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "clocks": clocks.summary(),
    }

    # end to end through the Python entry point
    e2e_steps = max(args.e2e_steps, K)
    if not args.no_e2e:
        if unequal:
            prompts = [torch.randint(0, V, (n,), generator=gen).tolist() for n in lengths]
        else:
            e2e_steps = min(e2e_steps, args.context - args.prompt - e2e_warmup - 2)
            prompts = [torch.randint(0, V, (e2e_prompt(e2e_steps),), generator=gen).tolist()
                       for _ in range(args.batch)]
        ev, h2d, d2h, n = e2e_run(prompts, e2e_steps)
        rec["e2e"] = {"value": round(ev, 1), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h,
                      "steps": n, "warmup": e2e_warmup}
    else:
        rec["e2e"] = {"value": 0.0, "unit": "tok/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0, "steps": 0}

    peak_tf = pk.get("bf16_tflops", FALLBACK_PEAKS["bf16_tflops"])
    if not args.no_points:
        # prefill: one 2,048-token prompt in one step (or, unequal workload, the whole batch's prompts in one step)
        plens = lengths if unequal else [2048]
        pms, T, flops, attn_flops = prefill_run(plens)
        rec["prefill"] = {"value": round(T / (pms / 1e3), 1), "tokens": T, "ms": round(pms, 3),
                          "frac": round(flops / (pms / 1e3) / 1e12 / peak_tf, 4)}
        if not unequal:
            points = {}
            for b in (1, 64):
                steps_b = max(64, min(K, 128))
                ms_b, _ = decode_run([start_ctx] * b, steps_b, max(W, 16))      # (the clocks settle, as for e2e)
                points[f"decode_b{b}"] = round(b * steps_b / (ms_b / 1e3), 1)
                if not args.no_e2e:
                    n_e2e = min(args.e2e_steps, args.context - args.prompt - e2e_warmup - 2)
                    prompts = [torch.randint(0, V, (e2e_prompt(n_e2e),), generator=gen).tolist() for _ in range(b)]
                    points[f"e2e_b{b}"] = round(e2e_run(prompts, n_e2e)[0], 1)
            if not args.no_e2e:
                # time to the first token of one request, host to host (the reference's tables quote it for a
                # short chat prompt, BENCHMARK.md:186-194): a 32-token and a 2,048-token prompt, best of five
                for n in (32, 2048):
                    if n + 2 > args.context:
                        continue
                    best = float("inf")
                    for _ in range(6):
                        prompt = torch.randint(0, V, (n,), generator=gen).tolist()
                        torch.cuda.synchronize()
                        t0 = time.perf_counter()
                        engine.generate([prompt], tq.GenerationParams.greedy(1, stop_token_ids=()))
                        best = min(best, time.perf_counter() - t0)
                    points[f"ttft_ms_p{n}"] = round(best * 1e3, 3)
            rec["points"] = points

    if not args.no_kernels:
        # device time by class of kernel: one decode step and the prefill, launched kernel by kernel
        graphs = engine.use_graphs
        engine.use_graphs = False
        try:
            slots = fill(ctx_lens)
            sampler = Sampler(tq.GenerationParams.greedy(1), args.batch, V, dev)
            tok = torch.randint(0, V, (args.batch,), generator=gen).tolist()

            def one_decode():
                logits = engine.step([StepRow(s, [t], [0]) for s, t in zip(slots, tok)], check=False)
                kernels.sample(logits, sampler.out)
                kernels.mark("sampler")

            one_decode()
            kern = class_table(timed_by_class(one_decode), "decode", nums, pk, tokens=args.batch,
                               cached_tokens=sum(ctx_lens) + 3 * args.batch, wanted_rows=args.batch, decode=True)
            for s in slots:
                engine.release(s)
            if not args.no_points:
                plens = lengths if unequal else [2048]
                ptoks = [torch.randint(0, V, (n,), generator=gen).tolist() for n in plens]
                held: list = []

                def one_prefill():
                    for s in held:
                        engine.release(s)
                    held[:] = [engine.new_sequence() for _ in plens]
                    engine.step([StepRow(s, t, [len(t) - 1]) for s, t in zip(held, ptoks)], check=False)

                one_prefill()
                attn = nums["attn_flops_per_key"] * sum(n * (n + 1) / 2 for n in plens)
                kern.update(class_table(timed_by_class(one_prefill), "prefill", nums, pk, tokens=sum(plens),
                                        cached_tokens=0, wanted_rows=len(plens), decode=False, attn_flops=attn))
                for s in held:
                    engine.release(s)
            engine.check_status()
            rec["kernels"] = kern
        finally:
            engine.use_graphs = graphs
    print(json.dumps(rec))
    return 0


if __name__ == "__main__":
    sys.exit(main())
