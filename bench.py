#!/usr/bin/env python3
"""Benchmark of the library's flagship step: decoding with the Qwen3-8B layer
sizes, random weights, bfloat16, on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one decode step of a batch of 8 sequences whose prompts are 2,048
tokens long (context length 4,096).  ``value`` is decoded tokens per second,
timed on the device with CUDA events over exactly K steps after W warm-up
steps; by default K extends the prompts to the full context (2,039 steps after
8 warm-up steps).  ``e2e`` is the same workload through ``Session.generate``
with host token ids in and out.  The line also carries a prefill measurement (one
2,048-token prompt), the decode step's memory roofline, decode at batch 1 and
64, and the SM clocks sampled during the timed region.

``--workload NAME`` runs another measurement instead and prints its own JSON: ``14b-unequal``, ``32b`` and
``long-context`` (larger Qwen3 sizes end to end), ``romepel`` / ``zevivik`` (those designs at two widths beside Qwen3
layers of equal size: a 2 048-token prompt, decode at batch 8, and every phase's time and roofline fraction), and
``pikalorn`` (that design at two widths beside Zevivik and Romepel layers of equal size, measured the same way),
``vodalorn`` (that design at two widths beside Pikalorn and Zevivik layers of equal size, measured the same way), ``gekilix`` (that design at two widths beside Zevivik and Romepel layers
of equal size, measured the same way), ``vuvalorn`` (that design at two widths beside Zevivik and Pikalorn layers of equal
size, measured the same way).
"""
from __future__ import annotations

import argparse
import json
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

QWEN3_8B = dict(architectures=["Qwen3ForCausalLM"], num_hidden_layers=36, hidden_size=4096, num_attention_heads=32,
                num_key_value_heads=8, head_dim=128, intermediate_size=12288, vocab_size=151936,
                rope_theta=1000000.0, rms_norm_eps=1e-6, tie_word_embeddings=False, attention_bias=False,
                max_position_embeddings=40960)
# The larger layer sizes of the benchmark description, for `--model 14b|32b` (not the default run).
SIZES = {
    "8b": {},
    "14b": dict(num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408),
    "32b": dict(num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600),
}
CONTEXT = 4096
PROMPT = 2048
BATCH = 8


def peaks() -> dict:
    p = ROOT / "MEASURED_PEAKS.json"
    if p.exists():
        try:
            d = json.loads(p.read_text())
            return {"hbm_gbs": float(d["hbm_gbs"]),
                    # the burst figure: the prefill step is 25 ms of work timed on its own, not a seconds-long loop
                    "bf16_tflops": float(d.get("bf16_tflops") or d["bf16_tflops_sustained"]),
                    "source": "measured"}
        except Exception:
            pass
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def sustained_tflops() -> float:
    p = ROOT / "MEASURED_PEAKS.json"
    try:
        return float(json.loads(p.read_text())["bf16_tflops_sustained"])
    except Exception:
        return 1400.0       # an earlier measurement on this pool: about 1.4 PFLOP/s at 1.3 GHz under the power cap


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.rows, self.proc, self.index = [], None, index

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.FIELDS}",
                                          "--format=csv,noheader,nounits", "-lms", "200"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def __exit__(self, *exc):
        if self.proc is not None:
            time.sleep(0.25)
            self.proc.terminate()
            self.thread.join(timeout=2)

    def summary(self) -> dict:
        sm = sorted(int(r[0]) for r in self.rows if r and r[0].isdigit())
        mx = [int(r[1]) for r in self.rows if len(r) > 1 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 2 + i and r[2 + i] == "Active" for r in self.rows)]
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(sm)}


def flops_prefill(cfg, T: int) -> float:
    """Multiply-adds times two of one T-token prompt: the layer matrices, causal
    attention (scores and weighted sum over half the square), one output row."""
    q = cfg.num_attention_heads * cfg.head_dim
    kv = cfg.num_key_value_heads * cfg.head_dim
    h, i = cfg.hidden_size, cfg.intermediate_size
    per_tok = 2.0 * (h * (q + 2 * kv) + q * h + 3 * h * i)
    attn = 4.0 * q * (T * (T + 1) / 2.0)
    return cfg.num_hidden_layers * (per_tok * T + attn) + 2.0 * h * cfg.vocab_size


def kv_bytes_per_token(cfg, esize: int = 2) -> int:
    return 2 * cfg.num_hidden_layers * cfg.num_key_value_heads * cfg.head_dim * esize


def timed_decode(engine, slots, first_tokens, steps: int, warmup: int):
    """W warm-up decode steps, then exactly K timed ones (greedy, token ids stay
    on the device).  Returns (milliseconds for K steps, mean kv length)."""
    import torch
    toks = engine.decode_run(slots, first_tokens, warmup) if warmup > 0 else None
    nxt = first_tokens if toks is None else toks[-1]
    torch.cuda.synchronize()
    lens0 = [engine.cache.length(s) for s in slots]
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    out = engine.decode_run(slots, nxt, steps)
    b.record()
    torch.cuda.synchronize()
    engine.model.rt.check_status()
    mean_len = sum(lens0) / len(lens0) + (steps + 1) / 2.0
    return a.elapsed_time(b), mean_len, out


def run_decode_point(model, cfg, batch: int, steps: int, warmup: int, seed: int = 0, with_phases: bool = False):
    import torch
    from nncpu_b200 import Engine
    per_seq = (CONTEXT + 63) // 64 * 64
    engine = Engine(model, max_tokens=per_seq * batch, max_seq_len=CONTEXT)
    g = torch.Generator().manual_seed(seed)
    prompts = torch.randint(0, cfg.vocab_size, (batch, PROMPT), generator=g).tolist()
    slots = [engine.alloc_slot() for _ in range(batch)]
    # prefill in chunks of sequences to bound activation memory
    firsts = []
    from nncpu_b200.kernels import ops
    for i in range(0, batch, 4):
        logits = engine.step(slots[i:i + 4], prompts[i:i + 4])
        ids = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
        ops.argmax(logits, ids)
        firsts += ids.tolist()
    steps = min(steps, CONTEXT - PROMPT - warmup - 1)
    ms, mean_len, _ = timed_decode(engine, slots, firsts, steps, warmup)
    tok_s = batch * steps / (ms / 1e3)
    bytes_step = model.weight_bytes_per_step() + batch * mean_len * kv_bytes_per_token(cfg)
    phases = None
    if with_phases:
        # the same engine, a few steps kernel by kernel under the phase profiler: where a step's time goes
        from nncpu_b200 import perf_enable, perf_reset, perf_totals
        for s in slots:      # the middle of the timed range, and in any case room for the steps below
            engine.cache.truncate(s, min(engine.cache.length(s), (PROMPT + CONTEXT) // 2, CONTEXT - 16))
        room = 9
        if room > 1:
            toks = [[1]] * batch
            engine.step(slots, toks)
            perf_enable(True)
            perf_reset()
            for _ in range(room - 1):
                engine.step(slots, toks)
            phases = {k: round(v["ms"] / (room - 1), 4) for k, v in perf_totals().items()}
            perf_enable(False)
            perf_reset()
    for s in slots:
        engine.free_slot(s)
    del engine
    torch.cuda.empty_cache()
    return tok_s, ms / steps, bytes_step, (mean_len - (steps + 1) / 2.0 + 1, mean_len + (steps + 1) / 2.0 - 1), phases


def run_prefill(model, cfg, reps: int = 3):
    import torch
    from nncpu_b200 import Engine
    engine = Engine(model, max_tokens=PROMPT + 64, max_seq_len=CONTEXT)
    g = torch.Generator().manual_seed(7)
    prompt = torch.randint(0, cfg.vocab_size, (PROMPT,), generator=g).tolist()
    best = None
    for r in range(reps + 1):
        slot = engine.alloc_slot()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        engine.step([slot], [prompt])
        b.record()
        torch.cuda.synchronize()
        engine.free_slot(slot)
        if r > 0:
            ms = a.elapsed_time(b)
            best = ms if best is None else min(best, ms)
    model.rt.check_status()
    del engine
    torch.cuda.empty_cache()
    return best


def run_e2e(model, cfg, steps: int, warmup: int):
    """The same decode workload through the public entry point: host token ids
    in, host token ids out, every step.  A first call of ``warmup`` steps on the
    same session is not timed (it builds the CUDA graph of this batch size)."""
    import torch
    from nncpu_b200 import GenerateParams, SamplerParams, Session, SessionParams
    session = Session(model, SessionParams(n_ctx=CONTEXT, seed=1, max_batch=BATCH))
    g = torch.Generator().manual_seed(3)
    prompts = torch.randint(0, cfg.vocab_size, (BATCH, PROMPT), generator=g).tolist()
    steps = min(steps, CONTEXT - PROMPT - 1)
    session.generate(prompts, GenerateParams(max_tokens=max(warmup, 1), sampler=SamplerParams.greedy()), stop_token_ids=())
    res = session.generate(prompts, GenerateParams(max_tokens=steps, sampler=SamplerParams.greedy()),
                           stop_token_ids=())
    n = sum(r.n_generated for r in res)
    decode_s = res[0].decode
    return {"value": n / decode_s if decode_s > 0 else None, "unit": "tokens/s",
            "h2d_bytes_per_step": session.engine.h2d_bytes_last_step, "d2h_bytes_per_step": 4 * BATCH,
            "prefill_s": res[0].prefill, "generated": n}


# The two larger workloads of the benchmark description, run through the public entry point, and a sweep of
# longer contexts than the contract's line covers.
WORKLOADS = {
    "14b-unequal": dict(model="14b", batch=16, prompt=(128, 2048), decode=256),
    "32b": dict(model="32b", batch=8, prompt=(2048, 2048), decode=512),
    "long-context": dict(model="8b"),
    "romepel": dict(model="8b"),
    "zevivik": dict(model="8b"),
    "pikalorn": dict(model="8b"),
    "vodalorn": dict(model="8b"),
    "gekilix": dict(model="8b"),
    "vuvalorn": dict(model="8b"),
}

# `--workload romepel`: the Romepel design (recurrent gla layers, windowed attention with a distance bias, sandwich
# norms, a dense xIELU feed-forward) at sizes that resemble a real model's layers, beside Qwen3 layers of equal width,
# depth, head counts, window and parameter count (a dense feed-forward of 1.5 x the gated one's width has its weights).
ROMEPEL_SIZES = {
    "2048": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, inter=6144, window=512, gla_heads=8, gla_dim=128,
                 gla_vdim=256, rank=32, vocab=32768),
    "4096": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, inter=12288, window=1024, gla_heads=16, gla_dim=128,
                 gla_vdim=256, rank=64, vocab=65536),
}


def romepel_configs(z: dict):
    """(Romepel configuration, the closest existing model's: Qwen3 with every layer on the same sliding window)."""
    from nncpu_b200.config import config_from_dict
    att = {"type": "attention", "mlp": {"kind": "dense", "ff": z["inter"] * 3 // 2},
           "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                     "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]}, "q_temp": {"coef": 0.25, "every": 256}}}
    gla = {"type": "gla", "mlp": {"kind": "dense", "ff": z["inter"] * 3 // 2},
           "mixer": {"heads": z["gla_heads"], "dim": z["gla_dim"], "vdim": z["gla_vdim"], "tau": 8.0, "rank": z["rank"]}}
    layers = [gla if i % 3 == 0 else att for i in range(z["layers"])]
    rom = config_from_dict({"architecture": "Romepel", "vocab": z["vocab"], "width": z["width"], "max_positions": CONTEXT,
                            "norm": {"eps": 1e-6}, "logit_softcap": 30.0, "layers": layers})
    qwen = config_from_dict(dict(QWEN3_8B, num_hidden_layers=z["layers"], hidden_size=z["width"],
                                 num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                                 intermediate_size=z["inter"], vocab_size=z["vocab"], use_sliding_window=True,
                                 sliding_window=z["window"], max_window_layers=0))
    return rom, qwen


# `--workload zevivik`: the Zevivik design (attention inside blocks of positions, latent attention, parallel blocks,
# routed experts with a shared one, a looped range of layers) at sizes that resemble a real model's layers, beside Qwen3
# layers of equal width, layer runs, head counts, span and active feed-forward width (top x expert + shared = gated).
ZEVIVIK_SIZES = {
    "2048": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, inter=6144, window=1024, lat_heads=16, lat_dim=128,
                 lat_vdim=128, rank=128, experts=16, top=2, vocab=32768),
    "4096": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, inter=12288, window=1024, lat_heads=16, lat_dim=128,
                 lat_vdim=256, rank=128, experts=16, top=2, vocab=65536),
}


def zevivik_configs(z: dict):
    """(Zevivik configuration, the closest existing model's: Qwen3 with every layer on a sliding window of the block's
    size).  Six layers of which the second and third run twice: eight layer runs, five of them with routed experts."""
    from nncpu_b200.config import config_from_dict
    dense = {"kind": "dense", "ff": z["inter"]}
    moe = {"kind": "moe", "expert": {"ff": z["inter"] // 4, "limit": 7.0}, "router": {"experts": z["experts"], "top": z["top"]},
           "shared": {"ff": z["inter"] // 2, "limit": 7.0}}
    def att(mlp):
        return {"type": "attention", "mlp": mlp,
                "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                          "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]}, "rot": {"base": 1000000.0, "dims": z["dim"]}}}
    def lat(mlp):
        return {"type": "latent_attention", "mlp": mlp,
                "mixer": {"heads": z["lat_heads"], "dim": z["lat_dim"], "vdim": z["lat_vdim"], "kv_rank": z["rank"],
                          "scale": z["lat_dim"] ** -0.5}}
    layers = [att(dense), att(moe), lat(moe), att(moe), lat(dense), att(dense)]
    zev = config_from_dict({"architecture": "Zevivik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0}, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": layers})
    qwen = config_from_dict(dict(QWEN3_8B, num_hidden_layers=z["layers"], hidden_size=z["width"],
                                 num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                                 intermediate_size=z["inter"], vocab_size=z["vocab"], use_sliding_window=True,
                                 sliding_window=z["window"], max_window_layers=0))
    return zev, qwen


# `--workload pikalorn`: the Pikalorn design (one-norm parallel layers; attention with sinks, values that are the keys
# and an output gate; latent attention with a query latent, a shared rotated key part and sinks, every other one of
# them reading the cache of the one before; the gated delta rule) at sizes that resemble a real model's layers, beside
# the two closest existing designs at equal width, depth, head counts and feed-forward width: Zevivik (attention and
# latent attention, where Pikalorn has a recurrent layer: attention) and Romepel (its recurrent gla layers at the places
# of the delta layers, attention elsewhere).
PIKALORN_SIZES = {
    "2048": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, inter=6144, lat_heads=16, lat_dim=64, rot_dim=64,
                 lat_vdim=128, rank=64, q_rank=768, delta_heads=16, delta_kv=8, delta_dim=128, delta_vdim=128, conv=4,
                 vocab=32768),
    "4096": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, inter=12288, lat_heads=32, lat_dim=64, rot_dim=64,
                 lat_vdim=128, rank=64, q_rank=1536, delta_heads=32, delta_kv=16, delta_dim=128, delta_vdim=128, conv=4,
                 vocab=65536),
}


def pikalorn_configs(z: dict):
    """(Pikalorn configuration, Zevivik's and Romepel's of equal size).  Eight layers: attention, latent, delta, latent
    on the second layer's cache, and the same four again."""
    from nncpu_b200.config import config_from_dict
    dense = {"kind": "dense", "ff": z["inter"]}
    rot = {"base": 1000000.0, "dims": z["dim"]}
    lrot = {"base": 10000.0, "dims": z["rot_dim"], "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}}

    def att():
        return {"type": "attention", "mlp": dense,
                "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                          "scale": z["dim"] ** -0.5, "rot": rot}}

    def lat(kv_from=None):
        m = {"heads": z["lat_heads"], "dim": z["lat_dim"], "rot_dim": z["rot_dim"], "vdim": z["lat_vdim"],
             "kv_rank": z["rank"], "q_rank": z["q_rank"], "scale": (z["lat_dim"] + z["rot_dim"]) ** -0.5, "rot": lrot}
        if kv_from is not None:
            m["kv_from"] = kv_from
        return {"type": "latent_attention", "mlp": dense, "mixer": m}

    def delta():
        return {"type": "delta", "mlp": dense,
                "mixer": {"heads": z["delta_heads"], "kv_heads": z["delta_kv"], "dim": z["delta_dim"],
                          "vdim": z["delta_vdim"], "conv": z["conv"]}}

    assert z["layers"] % 4 == 0
    layers = []
    for i in range(0, z["layers"], 4):
        layers += [att(), lat(), delta(), lat(kv_from=i + 1)]
    pik = config_from_dict({"architecture": "Pikalorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0}, "layers": layers})
    zatt = {"type": "attention", "mlp": dense,
            "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                      "scale": z["dim"] ** -0.5, "rot": rot}}
    zlat = {"type": "latent_attention", "mlp": dense,
            "mixer": {"heads": z["lat_heads"], "dim": z["lat_dim"] + z["rot_dim"], "vdim": z["lat_vdim"],
                      "kv_rank": z["rank"] + z["rot_dim"], "scale": (z["lat_dim"] + z["rot_dim"]) ** -0.5}}
    zev = config_from_dict({"architecture": "Zevivik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0}, "layers": [zatt, zlat] * (z["layers"] // 2)})
    ratt = {"type": "attention", "mlp": {"kind": "dense", "ff": z["inter"] * 3 // 2},
            "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                      "scale": z["dim"] ** -0.5}}
    rgla = {"type": "gla", "mlp": {"kind": "dense", "ff": z["inter"] * 3 // 2},
            "mixer": {"heads": z["delta_heads"], "dim": z["delta_dim"], "vdim": z["delta_vdim"], "tau": 8.0,
                      "rank": z["width"] // 64}}
    rom = config_from_dict({"architecture": "Romepel", "vocab": z["vocab"], "width": z["width"], "max_positions": CONTEXT,
                            "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
                            "layers": [rgla if i % 4 == 2 else ratt for i in range(z["layers"])]})
    return pik, zev, rom


# `--workload vodalorn`: the Vodalorn design (pre-norm layers with layer norms and a residual weight; pairs of windowed
# softmax attention and retention; the gated delta rule with a decay per key channel; the square of relu; experts chosen
# among the best groups; a hashed embedding of token pairs; a per-layer token input; a looped range of layers whose
# passes start from a product with the embedding output) at sizes that resemble a real model's layers, beside the two
# closest existing designs at equal width, layer runs, head counts and active feed-forward width: Pikalorn (attention
# where Vodalorn has a pair, its delta rule at the same places, gated feed-forwards) and Zevivik (a loop over the same
# range, routed experts of the same sizes at the same places, attention everywhere).
VODALORN_SIZES = {
    "2048": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, ret_heads=8, ret_dim=128, inter=6144,
                 delta_heads=16, delta_kv=8, delta_dim=128, delta_vdim=128, conv=4, rank=64, experts=16, top=2, groups=(4, 2),
                 side=128, buckets=65521, vocab=32768),
    "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, window=1024, ret_heads=16, ret_dim=128, inter=12288,
                 delta_heads=32, delta_kv=16, delta_dim=128, delta_vdim=128, conv=4, rank=128, experts=16, top=2, groups=(4, 2),
                 side=256, buckets=65521, vocab=65536),
}


def vodalorn_configs(z: dict):
    """(Vodalorn configuration, Pikalorn's and Zevivik's of equal size).  Five layers (pair + dense, delta + experts,
    pair + experts, pair + experts, delta + dense) of which the three in the middle run twice: eight layer runs."""
    from nncpu_b200.config import config_from_dict
    rot = {"base": 1000000.0, "dims": z["dim"]}
    # a token's active feed-forward width is the gated one's: experts of a quarter of it (three matrices each, the top
    # 2), and a dense one with two matrices of 1.5 times it
    moe = {"kind": "moe", "expert": {"ff": z["inter"] // 4, "limit": 7.0},
           "router": {"experts": z["experts"], "top": z["top"], "scale": 1.0, "groups": {"count": z["groups"][0], "keep": z["groups"][1]}}}
    dense = {"kind": "dense", "ff": z["inter"] * 3 // 2}

    def pair(mlp):
        return {"type": "parallel", "mlp": mlp,
                "mixer": {"left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                                   "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]}, "rot": rot},
                          "right": {"heads": z["ret_heads"], "dim": z["ret_dim"], "vdim": z["ret_dim"],
                                    "decay": [1.0 - 2.0 ** -(5 + i % 8) for i in range(z["ret_heads"])],
                                    "rot": {"base": 10000.0, "dims": z["ret_dim"]}}}}

    def delta(mlp):
        return {"type": "channel_delta", "mlp": mlp,
                "mixer": {"heads": z["delta_heads"], "kv_heads": z["delta_kv"], "dim": z["delta_dim"], "vdim": z["delta_vdim"],
                          "conv": z["conv"], "rank": z["rank"], "gate_rank": z["rank"]}}

    vod = config_from_dict({"architecture": "Vodalorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "residual_mult": 0.8, "token_side": {"dim": z["side"]},
                            "embedding": {"bigram": {"buckets": z["buckets"], "mul_prev": 8191, "mul_cur": 31}},
                            "loop": {"start": 1, "stop": 4, "times": 2},
                            "layers": [pair(dense), delta(moe), pair(moe), pair(moe), delta(dense)]})
    gated = {"kind": "dense", "ff": z["inter"]}
    patt = {"type": "attention", "mlp": gated,
            "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                      "scale": z["dim"] ** -0.5, "rot": rot}}
    pdel = {"type": "delta", "mlp": gated,
            "mixer": {"heads": z["delta_heads"], "kv_heads": z["delta_kv"], "dim": z["delta_dim"], "vdim": z["delta_vdim"],
                      "conv": z["conv"]}}
    pik = config_from_dict({"architecture": "Pikalorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0},
                            "layers": [patt, pdel, patt, patt, pdel, patt, patt, pdel]})
    zmoe = {"kind": "moe", "expert": {"ff": z["inter"] // 4, "limit": 7.0}, "router": {"experts": z["experts"], "top": z["top"]}}

    def zatt(mlp):
        return {"type": "attention", "mlp": mlp,
                "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                          "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]}, "rot": rot}}

    zev = config_from_dict({"architecture": "Zevivik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0}, "loop": {"start": 1, "stop": 4, "times": 2},
                            "layers": [zatt(gated), zatt(zmoe), zatt(zmoe), zatt(zmoe), zatt(gated)]})
    return vod, pik, zev


# `--workload gekilix`: the Gekilix design (state-space layers and windowed attention that keeps the first keys, routed
# experts with weighted inputs and a gated shared one) at sizes that resemble a real model's layers, beside the two
# closest existing designs at equal width and depth: Zevivik (the same experts in every layer, windowed attention
# everywhere) and Romepel (gla layers whose states have as many numbers at the state-space layers' places).
GEKILIX_SIZES = {
    "2048": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, vdim=128, window=1024, keep=64, inter=6144, experts=16, top=2,
                 ssm_heads=64, ssm_vdim=64, ssm_state=128, ssm_groups=4, conv=4, vocab=32768),
    "4096": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, vdim=128, window=1024, keep=64, inter=12288, experts=16, top=2,
                 ssm_heads=128, ssm_vdim=64, ssm_state=128, ssm_groups=8, conv=4, vocab=65536),
}


def gekilix_configs(z: dict):
    """(Gekilix configuration, Zevivik's and Romepel's of equal size).  Layers in fours: state space, attention, state
    space, state space.  Romepel's gla layers have heads of 128 x 256 for every four of 128 x 64."""
    from nncpu_b200.config import config_from_dict
    rot = {"base": 1000000.0, "dims": z["dim"]}
    experts = {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}}
    moe = dict(experts, expert={"ff": z["inter"] // 4}, shared={"ff": z["inter"] // 2})
    ssm = {"type": "mamba2", "mlp": moe,
           "mixer": {"heads": z["ssm_heads"], "vdim": z["ssm_vdim"], "state": z["ssm_state"], "groups": z["ssm_groups"],
                     "conv": z["conv"], "norm_groups": z["ssm_groups"]}}
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "scale": z["dim"] ** -0.5}
    gatt = {"type": "attention", "mlp": moe,
            "mixer": dict(att, mask={"size": z["window"], "keep_first": z["keep"]},
                          rot=dict(rot, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}))}
    gek = config_from_dict({"architecture": "Gekilix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "layers": [gatt if i % 4 == 1 else ssm for i in range(z["layers"])]})
    zmoe = dict(experts, expert={"ff": z["inter"] // 4, "limit": 7.0}, shared={"ff": z["inter"] // 2, "limit": 7.0})
    zatt = {"type": "attention", "mlp": zmoe, "mixer": dict(att, mask={"size": z["window"]}, rot=rot)}
    zev = config_from_dict({"architecture": "Zevivik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0}, "layers": [zatt] * z["layers"]})
    dense = {"kind": "dense", "ff": z["inter"] * 3 // 2}
    rgla = {"type": "gla", "mlp": dense,
            "mixer": {"heads": z["ssm_heads"] // 4, "dim": z["ssm_state"], "vdim": 4 * z["ssm_vdim"], "tau": 8.0,
                      "rank": z["width"] // 64}}
    ratt = {"type": "attention", "mlp": dense,
            "mixer": dict(att, mask={"size": z["window"]}, q_temp={"coef": 0.25, "every": 256})}
    rom = config_from_dict({"architecture": "Romepel", "vocab": z["vocab"], "width": z["width"], "max_positions": CONTEXT,
                            "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
                            "layers": [ratt if i % 4 == 1 else rgla for i in range(z["layers"])]})
    return gek, zev, rom


# `--workload vuvalorn`: the Vuvalorn design (convolved keys that are the values, capped scores, a gate per head, sandwich
# norms, clamped gated feed-forwards and experts some of which are the identity, a looped range of layers) at sizes that
# resemble a real model's layers, beside the two closest existing designs at equal width, layer runs and head counts, every
# key visible: Zevivik (the same feed-forwards and loop, experts without identities; a fused q/k/v epilogue) and Pikalorn
# (values that are the keys and a gate, dense feed-forwards).
VUVALORN_SIZES = {
    "2048": dict(width=2048, heads=16, kv_heads=4, dim=128, conv=4, inter=6144, experts=16, identity=4, top=2, vocab=32768),
    "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, conv=4, inter=12288, experts=16, identity=4, top=2, vocab=65536),
}


def vuvalorn_configs(z: dict):
    """(Vuvalorn configuration, Zevivik's and Pikalorn's of equal size).  Five layers of which the middle three run twice:
    eight layer runs, four of them with routed experts."""
    from nncpu_b200.config import config_from_dict
    rot = {"base": 1000000.0, "dims": z["dim"]}
    heads = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "rot": rot}
    router = {"experts": z["experts"], "top": z["top"]}
    loop = {"start": 1, "stop": 4, "times": 2}

    def model(architecture, mixer, dense, moe, **more):
        layers = [{"type": "attention", "mixer": mixer, "mlp": f} for f in (dense, moe, dense, moe, dense)]
        return config_from_dict({"architecture": architecture, "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                                 "embedding": {"scale": 1.0}, "layers": layers, **more})

    vuv = model("Vuvalorn", dict(heads, conv=z["conv"], softcap=30.0), {"kind": "dense", "ff": z["inter"], "limit": 7.0},
                {"kind": "moe", "expert": {"ff": z["inter"] // 2}, "router": dict(router, identity=z["identity"])}, loop=loop,
                logit_scale=0.5)
    zev = model("Zevivik", dict(heads, mask={"size": CONTEXT}), {"kind": "dense", "ff": z["inter"]},
                {"kind": "moe", "expert": {"ff": z["inter"] // 2, "limit": 7.0}, "router": router}, loop=loop)
    pik = config_from_dict({"architecture": "Pikalorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
                            "embedding": {"scale": 1.0},
                            "layers": [{"type": "attention", "mixer": heads, "mlp": {"kind": "dense", "ff": z["inter"]}}] * 8})
    return vuv, zev, pik


def phase_table(totals: dict, calls: int, pk: dict) -> dict:
    """Per phase of the profiler: milliseconds per step and, where the phase states its bytes and operations, the
    fraction of the roofline (the slower of bytes / copy bandwidth and operations / tensor throughput, over the time)."""
    out = {}
    for name, t in totals.items():
        ms = t["ms"] / calls
        row = {"ms": round(ms, 4)}
        ideal = max(t["bytes"] / calls / (pk["hbm_gbs"] * 1e9), t["flops"] / calls / (pk["bf16_tflops"] * 1e12))
        if ideal > 0 and ms > 0:
            row["roofline_frac"] = round(ideal / (ms / 1e3), 4)
        out[name] = row
    return out


def run_design_point(cfg, vocab: int, pk: dict, batch: int = 8, decode_steps: int = 128) -> dict:
    """One model: a 2 048-token prompt (best of 3 after a warm-up), then `decode_steps` device-timed greedy decode
    steps of `batch` sequences after 8 warm-up steps, then both kinds of step kernel by kernel under the phase profiler."""
    import torch
    from nncpu_b200 import Engine, Model, perf_enable, perf_reset, perf_totals
    from nncpu_b200.kernels import ops
    model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    g = torch.Generator().manual_seed(13)
    out = {"weight_bytes_per_step": model.weight_bytes_per_step()}
    engine = Engine(model, max_tokens=(PROMPT + 256) * batch, max_seq_len=PROMPT + 256, max_step_tokens=PROMPT)
    prompt = torch.randint(0, vocab, (PROMPT,), generator=g).tolist()
    best = None
    for r in range(4):
        slot = engine.alloc_slot()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        engine.step([slot], [prompt])
        b.record()
        torch.cuda.synchronize()
        engine.free_slot(slot)
        if r > 0:
            best = a.elapsed_time(b) if best is None else min(best, a.elapsed_time(b))
    out["prefill"] = {"tokens": PROMPT, "ms": round(best, 3), "tokens_per_s": round(PROMPT / (best / 1e3), 1)}
    slots = [engine.alloc_slot() for _ in range(batch)]
    firsts = []
    for s in slots:
        logits = engine.step([s], [torch.randint(0, vocab, (PROMPT,), generator=g).tolist()])
        ids = torch.empty(1, dtype=torch.int32, device=logits.device)
        ops.argmax(logits, ids)
        firsts += ids.tolist()
    ms, _, _ = timed_decode(engine, slots, firsts, decode_steps, 8)
    out["decode"] = {"batch": batch, "steps": decode_steps, "ms_per_step": round(ms / decode_steps, 4),
                     "tokens_per_s": round(batch * decode_steps / (ms / 1e3), 1),
                     "weights_hbm_frac": round(out["weight_bytes_per_step"] / (ms / decode_steps / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
    perf_enable(True)
    engine.step(slots, [[1]] * batch)
    perf_reset()
    for _ in range(4):
        engine.step(slots, [[1]] * batch)
    out["decode_phases"] = phase_table(perf_totals(), 4, pk)
    for s in slots:
        engine.free_slot(s)
    slot = engine.alloc_slot()
    engine.step([slot], [prompt])           # once kernel by kernel with the profiler on, not timed
    engine.free_slot(slot)
    slot = engine.alloc_slot()
    perf_reset()
    engine.step([slot], [prompt])
    out["prefill_phases"] = phase_table(perf_totals(), 1, pk)
    perf_enable(False)
    perf_reset()
    model.rt.check_status()
    del engine, model
    torch.cuda.empty_cache()
    return out


def run_romepel() -> dict:
    pk = peaks()
    out = {"workload": "romepel", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in ROMEPEL_SIZES.items():
        rom, qwen = romepel_configs(z)
        out["sizes"][name] = {"config": z, "romepel": run_design_point(rom, z["vocab"], pk),
                              "qwen3_same_size": run_design_point(qwen, z["vocab"], pk)}
    return out


def run_zevivik() -> dict:
    pk = peaks()
    out = {"workload": "zevivik", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in ZEVIVIK_SIZES.items():
        zev, qwen = zevivik_configs(z)
        out["sizes"][name] = {"config": z, "zevivik": run_design_point(zev, z["vocab"], pk),
                              "qwen3_same_size": run_design_point(qwen, z["vocab"], pk)}
    return out


def run_pikalorn() -> dict:
    pk = peaks()
    out = {"workload": "pikalorn", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in PIKALORN_SIZES.items():
        pik, zev, rom = pikalorn_configs(z)
        out["sizes"][name] = {"config": z, "pikalorn": run_design_point(pik, z["vocab"], pk),
                              "zevivik_same_size": run_design_point(zev, z["vocab"], pk),
                              "romepel_same_size": run_design_point(rom, z["vocab"], pk)}
    return out


def run_vodalorn() -> dict:
    pk = peaks()
    out = {"workload": "vodalorn", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in VODALORN_SIZES.items():
        vod, pik, zev = vodalorn_configs(z)
        out["sizes"][name] = {"config": z, "vodalorn": run_design_point(vod, z["vocab"], pk),
                              "pikalorn_same_size": run_design_point(pik, z["vocab"], pk),
                              "zevivik_same_size": run_design_point(zev, z["vocab"], pk)}
    return out


def run_gekilix() -> dict:
    pk = peaks()
    out = {"workload": "gekilix", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in GEKILIX_SIZES.items():
        gek, zev, rom = gekilix_configs(z)
        out["sizes"][name] = {"config": z, "gekilix": run_design_point(gek, z["vocab"], pk),
                              "zevivik_same_size": run_design_point(zev, z["vocab"], pk),
                              "romepel_same_size": run_design_point(rom, z["vocab"], pk)}
    return out


def run_vuvalorn() -> dict:
    pk = peaks()
    out = {"workload": "vuvalorn", "dtype": "bf16", "peaks": pk["source"], "prompt": PROMPT,
           "data": "synthetic: random weights, uniform random token ids", "sizes": {}}
    for name, z in VUVALORN_SIZES.items():
        vuv, zev, pik = vuvalorn_configs(z)
        out["sizes"][name] = {"config": z, "vuvalorn": run_design_point(vuv, z["vocab"], pk),
                              "zevivik_same_size": run_design_point(zev, z["vocab"], pk),
                              "pikalorn_same_size": run_design_point(pik, z["vocab"], pk)}
    return out


def run_long_context() -> dict:
    """Qwen3-8B sizes beyond the contract's 4 096 tokens: one prompt of 8 192 tokens, and decoding at batch 1 and 8
    with 16 384 and 32 768 keys per sequence (128 device-timed steps after 8 warm-up steps, greedy)."""
    import torch
    from nncpu_b200 import Engine, Model
    from nncpu_b200.config import config_from_dict
    from nncpu_b200.kernels import ops
    cfg = config_from_dict(dict(QWEN3_8B))
    model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    pk = peaks()
    out = {"workload": "long-context", "model": "Qwen3-8B sizes", "layers": cfg.num_hidden_layers, "dtype": "bf16",
           "peaks": pk["source"], "data": "synthetic: random weights, uniform random token ids"}
    g = torch.Generator().manual_seed(9)
    engine = Engine(model, max_tokens=8192 + 64, max_seq_len=8192 + 64, max_step_tokens=8192)
    prompt = torch.randint(0, cfg.vocab_size, (8192,), generator=g).tolist()
    best = None
    for r in range(3):
        slot = engine.alloc_slot()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        engine.step([slot], [prompt])
        b.record()
        torch.cuda.synchronize()
        engine.free_slot(slot)
        if r > 0:
            best = a.elapsed_time(b) if best is None else min(best, a.elapsed_time(b))
    out["prefill_8192"] = {"ms": best, "value": 8192 / (best / 1e3),
                           "frac": flops_prefill(cfg, 8192) / (best / 1e3) / (pk["bf16_tflops"] * 1e12)}
    del engine
    torch.cuda.empty_cache()
    for ctx in (16384, 32768):
        for batch in (1, 8):
            engine = Engine(model, max_tokens=(ctx + 256) * batch, max_seq_len=ctx + 256, max_step_tokens=8192)
            slots = [engine.alloc_slot() for _ in range(batch)]
            firsts = []
            for s in slots:          # prompts go in one by one, 8 192 tokens a step
                toks = torch.randint(0, cfg.vocab_size, (ctx,), generator=g).tolist()
                for at in range(0, ctx, 8192):
                    logits = engine.step([s], [toks[at:at + 8192]])
                ids = torch.empty(1, dtype=torch.int32, device=logits.device)
                ops.argmax(logits, ids)
                firsts += ids.tolist()
            ms, mean_len, _ = timed_decode(engine, slots, firsts, 128, 8)
            step_bytes = model.weight_bytes_per_step() + batch * mean_len * kv_bytes_per_token(cfg)
            out[f"decode_b{batch}_ctx{ctx}"] = {"value": batch * 128 / (ms / 1e3), "ms_per_step": ms / 128,
                                                "hbm_frac": step_bytes / (ms / 128 / 1e3) / 1e9 / pk["hbm_gbs"]}
            for s in slots:
                engine.free_slot(s)
            del engine
            torch.cuda.empty_cache()
    return out


def run_workload(name: str) -> dict:
    """Batch of prompts (lengths uniform in the workload's range) through
    ``Session.generate``: one prefill step, then the workload's decode steps,
    greedy, host token ids in and out.  The first call (a few tokens) builds the
    CUDA graphs and is not timed."""
    import torch
    from nncpu_b200 import GenerateParams, Model, SamplerParams, Session, SessionParams
    from nncpu_b200.config import config_from_dict
    w = WORKLOADS[name]
    cfg = config_from_dict(dict(QWEN3_8B, **SIZES[w["model"]]))
    model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    g = torch.Generator().manual_seed(5)
    lo, hi = w["prompt"]
    lengths = torch.randint(lo, hi + 1, (w["batch"],), generator=g).tolist()
    prompts = [torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist() for n in lengths]
    session = Session(model, SessionParams(n_ctx=hi + w["decode"] + 1, seed=1, max_batch=w["batch"]))
    session.generate(prompts, GenerateParams(max_tokens=4, sampler=SamplerParams.greedy()), stop_token_ids=())
    res = session.generate(prompts, GenerateParams(max_tokens=w["decode"], sampler=SamplerParams.greedy()),
                           stop_token_ids=())
    n = sum(r.n_generated for r in res)
    mean_len = sum(lengths) / len(lengths) + w["decode"] / 2.0
    step_bytes = model.weight_bytes_per_step() + w["batch"] * mean_len * kv_bytes_per_token(cfg)
    step_s = res[0].decode / w["decode"]
    pk = peaks()
    return {"workload": name, "model": f"Qwen3-{w['model'].upper()} sizes", "layers": cfg.num_hidden_layers,
            "batch": w["batch"], "prompt_tokens": sum(lengths), "prompt_lengths": f"{min(lengths)}..{max(lengths)}",
            "decode_steps": w["decode"], "generated": n, "prefill_s": res[0].prefill,
            "prefill_tokens_per_s": sum(lengths) / res[0].prefill, "decode_s": res[0].decode,
            "decode_tokens_per_s": n / res[0].decode, "ms_per_step": step_s * 1e3,
            "hbm_frac": step_bytes / step_s / 1e9 / pk["hbm_gbs"], "peaks": pk["source"], "dtype": "bf16",
            "data": "synthetic: random weights, uniform random token ids"}


def fp32_check(cfg, name: str) -> dict:
    """The same random weights (rounded to bfloat16) run in bfloat16 and in true float32: how far the
    logits of a 96-token prompt, and of 8 tokens decoded after it, are apart."""
    import torch
    from nncpu_b200 import Engine, Model
    from nncpu_b200.engine.model import parameter_list
    from nncpu_b200.parts import Runtime
    from nncpu_b200.weights import random_tensors_on_device
    g = torch.Generator().manual_seed(11)
    toks = torch.randint(0, cfg.vocab_size, (104,), generator=g).tolist()
    out = {}
    for dtype in ("bfloat16", "float32"):
        rt = Runtime("cuda:0", torch.bfloat16 if dtype == "bfloat16" else torch.float32)
        tensors = random_tensors_on_device(parameter_list(cfg.model_spec()), 0, torch.bfloat16, rt.device)
        if dtype == "float32":
            tensors = {k: v.float() for k, v in tensors.items()}
        model = Model(cfg, tensors, rt)
        del tensors
        engine = Engine(model, max_tokens=128)
        slot = engine.alloc_slot()
        rows = [engine.step([slot], [toks[:96]], [[0, 47, 95]]).clone()]
        rows += [engine.step([slot], [[t]]).clone() for t in toks[96:]]
        out[dtype] = torch.cat(rows).cpu()
        model.rt.check_status()
        del engine, model
        torch.cuda.empty_cache()
    diff = (out["bfloat16"] - out["float32"]).abs().max().item()
    scale = out["float32"].abs().max().item()
    agree = (out["bfloat16"].argmax(-1) == out["float32"].argmax(-1)).float().mean().item()
    return {"check": "bfloat16 against float32 logits", "model": f"Qwen3-{name.upper()} sizes",
            "layers": cfg.num_hidden_layers, "rows": out["float32"].shape[0], "max_abs_diff": diff,
            "max_abs_logit": scale, "relative": diff / scale, "same_top_token": agree}


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=CONTEXT - PROMPT)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=0, help="run fewer layers than the configuration has (named in config)")
    ap.add_argument("--skip-points", action="store_true")
    ap.add_argument("--model", default="8b", choices=sorted(SIZES), help="layer sizes (default: the benchmark's 8b)")
    ap.add_argument("--workload", choices=sorted(WORKLOADS),
                    help="instead of the contract's line: one of the description's larger workloads, end to end")
    ap.add_argument("--fp32-check", action="store_true",
                    help="instead of timing: logits of a short prompt in bfloat16 against the true 32-bit path")
    ap.add_argument("--no-launch-overlap", action="store_true",
                    help="for comparison: every kernel of a decode step waits for the end of the one before it")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "ZacWalk/nncpu is a Rust crate with no Python package and no Rust toolchain is installed: "
                          "pip cannot install it offline and it has no GPU path"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this library is single-GPU by design, --gpus {args.gpus} is not supported")
        return 2
    args.warmup = max(args.warmup, 3)

    import torch
    from nncpu_b200.config import config_from_dict
    from nncpu_b200 import Model
    from nncpu_b200.kernels import ops

    if args.no_launch_overlap:
        ops.launch_overlap(False)
    d = dict(QWEN3_8B, **SIZES[args.model])
    full_layers = d["num_hidden_layers"]
    if args.layers:
        d["num_hidden_layers"] = args.layers
    cfg = config_from_dict(d)
    pk = peaks()
    if args.fp32_check:
        print(json.dumps(fp32_check(cfg, args.model)))
        return 0
    if args.workload:
        special = {"long-context": run_long_context, "romepel": run_romepel, "zevivik": run_zevivik,
                   "pikalorn": run_pikalorn, "vodalorn": run_vodalorn, "gekilix": run_gekilix, "vuvalorn": run_vuvalorn}
        print(json.dumps(special[args.workload]() if args.workload in special else run_workload(args.workload)))
        return 0
    model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")

    prefill_ms = run_prefill(model, cfg)
    pf_flops = flops_prefill(cfg, PROMPT)
    launches0 = ops.launch_count()
    with ClockSampler() as clocks:
        tok_s, ms_step, bytes_step, key_range, phases = run_decode_point(model, cfg, BATCH, args.steps, args.warmup,
                                                                          with_phases=True)
    launches = ops.launch_count() - launches0
    points, points_frac = {}, {}
    if not args.skip_points:
        for name, batch in (("decode_b1", 1), ("decode_b64", 64)):
            point = run_decode_point(model, cfg, batch, args.steps, args.warmup)
            points[name] = point[0]
            # the same roofline as the headline's: used weights once and the live requests' cache, over the step's time
            points_frac[name] = round(point[2] / (point[1] / 1e3) / 1e9 / pk["hbm_gbs"], 4)
    e2e = run_e2e(model, cfg, args.steps, args.warmup)
    achieved = bytes_step / (ms_step / 1e3) / 1e9
    line = {
        "metric": f"decode tokens/s, Qwen3-{args.model.upper()} sizes, bf16, batch 8, 2048-token prompts, context 4096 "
                  f"(timed steps read {int(key_range[0])} to {int(key_range[1])} keys per sequence)",
        "value": tok_s, "unit": "tokens/s", "n_gpus": 1, "steps": min(args.steps, CONTEXT - PROMPT - args.warmup - 1),
        "warmup": args.warmup, "ms_per_step": ms_step, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random weights, uniform random token ids",
        "impl": "ours",
        "config": {"model": f"Qwen3-{args.model.upper()} sizes", "layers": cfg.num_hidden_layers, "layers_of_config": full_layers,
                   "hidden_size": cfg.hidden_size, "heads": cfg.num_attention_heads,
                   "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate_size": cfg.intermediate_size, "vocab_size": cfg.vocab_size,
                   "global_batch": BATCH, "seq_len": CONTEXT, "prompt_len": PROMPT, "parallelism": "single GPU",
                   "l2": "inputs larger than L2 (15 GB of weights per step)", "peaks": pk["source"],
                   "keys_first_timed_step": int(key_range[0]), "keys_last_timed_step": int(key_range[1])},
        "e2e": e2e,
        "gpu_launches": launches,
        "prefill": {"value": PROMPT / (prefill_ms / 1e3), "tokens": PROMPT, "ms": prefill_ms,
                    "frac": pf_flops / (prefill_ms / 1e3) / (pk["bf16_tflops"] * 1e12)},
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": achieved / pk["hbm_gbs"]},
        "points": points,
        "points_roofline_frac": points_frac,
        "phases": {"unit": "ms per decode step, kernel by kernel under the phase profiler (not the graph)",
                   **(phases or {})},
        "prefill_batched": {"tokens": BATCH * PROMPT, "ms": e2e["prefill_s"] * 1e3,
                            "value": BATCH * PROMPT / e2e["prefill_s"],
                            "frac_of_sustained": BATCH * pf_flops / e2e["prefill_s"] / (sustained_tflops() * 1e12),
                            "note": "the 8 prompts of the end-to-end run as one step, host work included; 0.2 s of dense "
                                    "products run under the power cap, so its fraction is taken against the sustained "
                                    "figure of the measured peaks, where the single prompt's 25 ms run at burst clocks"},
        "clocks": clocks.summary(),
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
