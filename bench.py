#!/usr/bin/env python3
"""Headline benchmark: decode tokens per second at Llama-3-8B layer sizes with random weights
on one B200, plus the prefill of 2,048 tokens, the decode roofline and the end-to-end number
through the Python entry point.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--batch B] [--context T]

Prints ONE JSON line.  A "step" is one decode step of the whole batch.  ``value`` is timed on
the device with CUDA events around K steps of the step function plus the sampling kernel;
``e2e`` is the same through ``LLM.submit``/``LLM.step`` with host token ids in (pinned memory,
one copy per step) and the chosen tokens read back to the host every step.
"""

from __future__ import annotations

import argparse
import json
import statistics
import sys
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

from baseline.common import (SIZE_LABELS, SIZES_BY_NAME, ClockSampler, kv_bytes_per_token,
                             model_config, peaks, prefill_flops, spread, weight_bytes)

# the headline configuration: Llama-3-8B layer sizes
SIZES = SIZES_BY_NAME["llama-3-8b"]
#: up to this many layers the random model is written as a model folder and opened through
#: ``load_model`` like any user's; above, each tensor is drawn on the device when the model
#: asks for it (a folder of 16 GB takes minutes to draw on the CPU and to write)
FOLDER_MAX_LAYERS = 4


def build_engine(n_layers: int, capacity_tokens: int, max_requests: int, page_size: int,
                 sizes: dict | None = None):
    """The engine with random weights N(0, 0.02): (config, model, LLM, how the weights came)."""
    import tempfile

    import torch

    from scratch_llm_b200.config import config_from_dict
    from scratch_llm_b200.engine import LLM, build_model, load_model
    from scratch_llm_b200.kernels import ops
    from scratch_llm_b200.parts import BuildContext
    from scratch_llm_b200.weights import write_random_model
    from scratch_llm_b200.weights.random_init import random_tensors

    cfg = config_from_dict({**(sizes or SIZES), "num_hidden_layers": n_layers,
                            "architectures": ["LlamaForCausalLM"]})
    if n_layers <= FOLDER_MAX_LAYERS:
        # the way a user's model comes in: a folder with config.json and model.safetensors
        with tempfile.TemporaryDirectory() as tmp:
            write_random_model(cfg, tmp, seed=0)
            model = load_model(tmp, "bfloat16", verbose=False)
        how = "model folder (config.json + model.safetensors) through load_model"
    else:
        model = build_model(cfg)
        ops.prepare(model.head_dims(), verbose=False)
        specs = model.param_specs()
        device = torch.device("cuda", 0)

        class Lazy(dict):
            """Draws each tensor on the device when the model asks for it, so that the random
            weights never exist twice."""

            def __missing__(self, name):
                return random_tensors({name: specs[name]}, 0, torch.bfloat16, device=device)[name]

        model.load(Lazy(), BuildContext(dtype=torch.bfloat16, device=device))
        model.config = cfg
        how = "drawn on the device tensor by tensor (no folder of this size is written)"
    llm = LLM(model, max_tokens=capacity_tokens, page_size=page_size, max_requests=max_requests,
              max_batch_tokens=4096, chunk_size=2048)
    return cfg, model, llm, how


#: --compare nilevik: layer sizes that resemble real models' (four layers each: attention,
#: attention, delta rule, attention, every one with a feed-forward), and the Llama-style model of
#: the same width, heads, head size, feed-forward width, vocabulary and layer count beside them
COMPARE_SIZES = {
    "1b-like": dict(width=2048, heads=32, kv_heads=8, dim=64, ff=8192, vocab=32768, window=1024,
                    side_dim=64, delta=dict(heads=16, kv_heads=8, dim=128, vdim=128, conv=4)),
    "8b-like": dict(width=4096, heads=32, kv_heads=8, dim=128, ff=14336, vocab=32768, window=1024,
                    side_dim=128, delta=dict(heads=32, kv_heads=16, dim=128, vdim=128, conv=4)),
}


def compare_configs(name: str):
    """(Nilevik config, Llama config) of equal size."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    mlp = {"kind": "dense", "ff": z["ff"]}
    attention = {"type": "attention", "mlp": mlp, "mixer": {
        "heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
        "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]},
        "q_temp": {"coef": 0.25, "every": 256}}}
    delta = {"type": "delta", "mlp": mlp, "mixer": dict(z["delta"])}
    nilevik = config_from_dict({
        "architecture": "Nilevik", "vocab": z["vocab"], "width": z["width"],
        "norm": {"eps": 1e-5}, "token_side": {"dim": z["side_dim"]},
        "layers": [attention, attention, delta, attention], "max_position": 8192})
    llama = config_from_dict({
        "architectures": ["LlamaForCausalLM"], "hidden_size": z["width"], "num_hidden_layers": 4,
        "num_attention_heads": z["heads"], "num_key_value_heads": z["kv_heads"],
        "head_dim": z["dim"], "intermediate_size": z["ff"], "vocab_size": z["vocab"],
        "tie_word_embeddings": True, "max_position_embeddings": 8192})
    return nilevik, llama


def vobosun_config(name: str):
    """The Vobosun design at the sizes of COMPARE_SIZES: attention (dense feed-forward), the
    generalized delta rule (routed feed-forward), attention (routed), attention (dense).  The
    recurrent layer has heads of 64 across the width; a routed feed-forward has 16 experts of a
    quarter of the dense size of which a token uses 2, four identity experts, four groups of which
    two are kept, and a shared expert of the same quarter."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    dense = {"kind": "dense", "ff": z["ff"]}
    routed = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "shared": {"ff": z["ff"] // 4},
              "router": {"experts": 16, "identity": 4, "top": 2, "groups": {"count": 4, "keep": 2}}}
    mixer = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
             "scale": z["dim"] ** -0.5,
             "rot": {"base": 1000000.0, "dims": z["dim"], "scaling": {"factor": 8.0}}}
    delta = {"heads": z["width"] // 64, "dim": 64, "decay_rank": 64}
    return config_from_dict({
        "architecture": "Vobosun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
        "max_position": 8192,
        "layers": [{"type": "attention", "mixer": mixer, "mlp": dense},
                   {"type": "general_delta", "mixer": delta, "mlp": routed},
                   {"type": "attention", "mixer": mixer, "mlp": routed},
                   {"type": "attention", "mixer": mixer, "mlp": dense}]})


def titedra_config(name: str):
    """The Titedra design at the sizes of COMPARE_SIZES: four layers of latent attention (as many
    heads, the head size as the unrotated part, a rotated part of 64, a query latent of three
    quarters of the width, a key/value latent of 192: the cached vector has 256 entries, the
    largest the tensor-core attention kernels take), with a dense, two routed and a dense
    feed-forward.  A routed one has 16 ungated experts of a quarter of the dense size in four
    groups of which two are kept, and a token uses 4.  The two middle layers form a loop of one
    pass, so that the stream is joined with the embedding output once and as many layers run as
    in the models beside it."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    dense = {"kind": "dense", "ff": z["ff"]}
    routed = {"kind": "moe", "expert": {"ff": z["ff"] // 4},
              "router": {"experts": 16, "top": 4, "groups": {"count": 4, "keep": 2}}}
    mixer = {"heads": z["heads"], "dim": z["dim"], "rot_dim": 64, "vdim": z["dim"],
             "q_rank": 3 * z["width"] // 4, "kv_rank": 192, "scale": (z["dim"] + 64) ** -0.5,
             "rot": {"base": 1000000.0, "dims": 64}}
    return config_from_dict({
        "architecture": "Titedra", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.0}, "logit_scale": 1.0, "max_position": 8192,
        "loop": {"start": 1, "stop": 3, "times": 1},
        "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": mlp}
                   for mlp in (dense, routed, routed, dense)]})


def tubevik_config(name: str):
    """The Tubevik design at the sizes of COMPARE_SIZES: attention (window, cap, gate per head),
    two mixers side by side (attention in chunks of the window's length with half as many heads
    beside the delta rule of COMPARE_SIZES with a decay per key channel), attention that borrows
    the first layer's keys and values, and the two mixers side by side again; every layer with a
    clamped gated feed-forward of the dense size."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    mlp = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    rot = {"base": 2000000.0, "dims": z["dim"],
           "scaling": {"factor": 4.0, "original": 2048, "fast": 16.0, "slow": 2.0}}
    attention = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                 "scale": z["dim"] ** -0.5, "softcap": 50.0, "mask": {"size": z["window"]},
                 "rot": rot}
    left = {"heads": z["heads"] // 2, "kv_heads": z["kv_heads"] // 2, "dim": z["dim"],
            "vdim": z["dim"], "scale": 1.0, "mask": {"size": z["window"]},
            "rot": {"base": 100000.0, "dims": z["dim"] // 2}}
    both = {"left": left, "right": dict(z["delta"]), "left_scale": 0.7, "right_scale": 1.3}
    return config_from_dict({
        "architecture": "Tubevik", "vocab": z["vocab"], "width": z["width"],
        "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_softcap": 40.0, "max_position": 8192,
        "layers": [{"type": "attention", "mixer": attention, "mlp": mlp},
                   {"type": "parallel", "mixer": both, "mlp": mlp},
                   {"type": "attention", "mixer": dict(attention, kv_from=0), "mlp": mlp},
                   {"type": "parallel", "mixer": both, "mlp": mlp}]})


def deganex_config(name: str):
    """The Deganex design at the sizes of COMPARE_SIZES: a state-space layer (twice the width in
    heads of 64, state 128), latent attention (as many heads, the head size as the unrotated
    part, a rotated part of 64, a latent of 192: the cached vector has 256 entries, the largest
    the tensor-core attention kernels take), a matrix memory (keys of 256, values of 512, one
    head per 512 of the width) and latent attention again; every layer with a routed
    feed-forward of 16 experts and a gated shared one, each a quarter of the dense size, of which
    a token uses 3 and the shared one: as much as the dense feed-forward."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    d = z["width"]
    mlp = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": 16, "top": 3},
           "shared": {"ff": z["ff"] // 4}}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": z["heads"], "dim": z["dim"], "rot_dim": 64, "vdim": z["dim"], "kv_rank": 192,
        "scale": (z["dim"] + 64) ** -0.5, "rot": {"base": 1000000.0, "dims": 64}}}
    state_space = {"type": "mamba2", "mlp": mlp, "mixer": {
        "heads": 2 * d // 64, "vdim": 64, "state": 128, "groups": 4, "conv": 4, "norm_groups": 4}}
    memory = {"type": "mlstm", "mlp": mlp, "mixer": {
        "heads": d // 512, "dim": 256, "vdim": 512, "gate_cap": 20.0}}
    return config_from_dict({
        "architecture": "Deganex", "vocab": z["vocab"], "width": d, "norm": {"eps": 1e-5},
        "logit_softcap": 25.0, "max_position": 8192,
        "embedding": {"bigram": {"buckets": 65521, "mul_prev": 4099, "mul_cur": 257}},
        "layers": [state_space, latent, memory, latent]})


def kumudra_config(name: str):
    """The Kumudra design at the sizes of COMPARE_SIZES: two streams; attention (half of the heads,
    window, biases, a quarter of each head rotated) beside time mixing (heads of 64 across the
    width) with a dense feed-forward, gated linear attention (keys of 128, values of 256, one head
    per 256 of the width) and lightning attention (heads of 128 across the width) with a routed
    one of 16 experts, each a quarter of the dense size, of which a token uses 4, and the two
    mixers side by side again with a dense one."""
    from scratch_llm_b200.config import config_from_dict

    z = COMPARE_SIZES[name]
    d = z["width"]
    dense = {"kind": "dense", "ff": z["ff"]}
    routed = {"kind": "moe", "expert": {"ff": z["ff"] // 4},
              "router": {"experts": 16, "top": 4, "scale": 1.3}}
    left = {"heads": z["heads"] // 2, "kv_heads": z["kv_heads"] // 2, "dim": z["dim"],
            "vdim": z["dim"], "scale": z["dim"] ** -0.5, "mask": {"size": z["window"]},
            "rot": {"base": 500000.0, "dims": z["dim"] // 4,
                    "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 4096}}}
    both = {"type": "parallel", "mlp": dense, "mixer": {
        "left": left, "right": {"heads": d // 64, "dim": 64}, "left_scale": 0.7,
        "right_scale": 1.1}}
    gla = {"type": "gla", "mlp": routed, "mixer": {"heads": d // 256, "dim": 128, "vdim": 256,
                                                   "tau": 16.0}}
    heads = d // 128
    lightning = {"type": "lightning", "mlp": routed, "mixer": {
        "heads": heads, "dim": 128, "vdim": 128,
        "decay": [1.0 - 2.0 ** (-2.0 - 8.0 * h / heads) for h in range(heads)]}}
    return config_from_dict({
        "architecture": "Kumudra", "vocab": z["vocab"], "width": d, "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.5}, "residual_mult": 0.8, "streams": 2, "max_position": 8192,
        "layers": [both, gla, lightning, both]})


#: low ranks that only a model's tensors say (a size of -1 in a parameter's shape): random
#: weights are drawn with this one
RANDOM_LOW_RANK = 64


def engine_of(cfg, capacity_tokens: int, max_requests: int, page_size: int):
    """An engine for ``cfg`` with random weights drawn on the device, tensor by tensor."""
    import torch

    from scratch_llm_b200.engine import LLM, build_model
    from scratch_llm_b200.kernels import ops
    from scratch_llm_b200.parts import BuildContext
    from scratch_llm_b200.weights.random_init import random_tensors

    model = build_model(cfg)
    jobs = model.kernel_jobs(torch.bfloat16)
    if jobs is None:
        ops.prepare(model.head_dims(), verbose=False)
    else:
        ops.prepare_jobs(jobs, verbose=False)
    specs = model.param_specs()
    device = torch.device("cuda", 0)

    class Lazy(dict):
        def __missing__(self, name):
            spec = specs[name]
            if -1 in spec.shape:
                spec = type(spec)(tuple(RANDOM_LOW_RANK if n == -1 else n for n in spec.shape),
                                  spec.kind)
            return random_tensors({name: spec}, 0, torch.bfloat16, device=device)[name]

    model.load(Lazy(), BuildContext(dtype=torch.bfloat16, device=device))
    model.config = cfg
    return LLM(model, max_tokens=capacity_tokens, page_size=page_size, max_requests=max_requests,
               max_batch_tokens=4096, chunk_size=2048)


def compare_main(args) -> int:
    """--compare nilevik | vobosun | titedra | tubevik | deganex | kumudra: prefill and decode throughput of
    that design beside the engine's other models of equal size (for Vobosun: Nilevik, the closest one, a hybrid of
    attention and a delta rule with normed branch outputs, and the Llama-style model; for
    Titedra: Vobosun, the closest one, with norms around every branch, a partly rotated
    attention and routed experts, and the Llama-style model; for Tubevik: Nilevik, the closest one, likewise a hybrid of windowed
    attention and a gated delta rule, and the Llama-style model; for Deganex: Titedra, the closest
    one, with latent attention and routed experts, Nilevik for its recurrence, and the
    Llama-style model; for Kumudra: Tubevik, the closest one, with attention beside a recurrence
    with a decay per key channel, Deganex for its scan and routed experts, and the Llama-style
    model), at the sizes of COMPARE_SIZES.
    One JSON line."""
    import torch

    torch.cuda.set_device(0)
    names = [args.compare_sizes] if args.compare_sizes else list(COMPARE_SIZES)
    out = {"compare": args.compare, "dtype": "bf16", "data": "synthetic", "batch": args.batch,
           "context": args.context, "prefill_tokens": args.prefill_tokens, "steps": args.steps,
           "warmup": args.warmup, "sizes": {}}
    capacity = args.batch * (args.context + args.warmup + args.steps + 64) + 2 * args.prefill_tokens
    with torch.no_grad():
        for name in names:
            out["sizes"][name] = entry = {"layers": "attention, attention, delta, attention",
                                          **{k: v for k, v in COMPARE_SIZES[name].items()}}
            archs = list(zip(("nilevik", "llama"), compare_configs(name)))
            if args.compare in ("vobosun", "titedra"):
                entry["vobosun_layers"] = ("attention + dense, general_delta + routed, "
                                           "attention + routed, attention + dense")
                archs.insert(0, ("vobosun", vobosun_config(name)))
            if args.compare == "tubevik":
                entry["tubevik_layers"] = ("attention + dense, (chunked attention | delta rule) "
                                           "+ dense, attention on the first layer's keys + dense, "
                                           "(chunked attention | delta rule) + dense")
                archs.insert(0, ("tubevik", tubevik_config(name)))
            if args.compare == "titedra":
                entry["titedra_layers"] = ("latent_attention + dense, 2 x (latent_attention + "
                                           "routed) as a loop of one pass, latent_attention + "
                                           "dense")
                archs = [("titedra", titedra_config(name))] + \
                    [a for a in archs if a[0] != "nilevik"]
            if args.compare == "deganex":
                entry["deganex_layers"] = ("state space, latent attention, matrix memory, latent "
                                           "attention, each + routed with a shared expert")
                archs[:0] = [("deganex", deganex_config(name)), ("titedra", titedra_config(name))]
            if args.compare == "kumudra":
                entry["kumudra_layers"] = ("(windowed attention | time mixing) + dense, gated "
                                           "linear attention + routed, lightning attention + "
                                           "routed, (windowed attention | time mixing) + dense")
                archs = [("kumudra", kumudra_config(name)), ("tubevik", tubevik_config(name)),
                         ("deganex", deganex_config(name))] + [a for a in archs if a[0] == "llama"]
            for arch, cfg in archs:
                llm = engine_of(cfg, capacity, args.batch + 1, args.page_size)
                with ClockSampler(0) as clk:
                    prefill = statistics.median(time_prefill(llm, cfg, args.prefill_tokens, reps=5))
                    ms, launches, per_step = time_decode_device(
                        llm, cfg, args.batch, args.context, args.steps, args.warmup, arch[0])
                entry[arch] = {
                    "prefill_tok_s": round(args.prefill_tokens / prefill * 1e3, 1),
                    "prefill_ms": round(prefill, 3),
                    "decode_tok_s": round(args.batch / ms * 1e3, 1), "decode_ms": round(ms, 4),
                    "decode_spread": spread(per_step), "gpu_launches": launches,
                    "clocks": clk.summary}
                del llm
                torch.cuda.empty_cache()
    print(json.dumps(out))
    return 0


def time_serve(llm, cfg, n_requests: int, seed: int = 3):
    """The baseline's continuous-batching workload: `n_requests` requests with prompt lengths
    16-2048 and output lengths 16-512 (seeded, uniform), all queued at once, through LLM.serve
    (host token ids in and out).  Returns (generated tok/s, prompt tokens, generated tokens,
    seconds, steps)."""
    import random

    from scratch_llm_b200 import Request, SamplingParams

    rng = random.Random(seed)
    reqs = []
    for i in range(n_requests):
        n_in, n_out = rng.randint(16, 2048), rng.randint(16, 512)
        reqs.append(Request(f"s{i}", [rng.randrange(cfg.vocab_size) for _ in range(n_in)],
                            SamplingParams(temperature=0.0, max_tokens=n_out)))
    llm.serve(reqs[:4])          # warm-up: compiles nothing, but pages in the kernels
    res = llm.serve(reqs)
    n_out = sum(len(c.token_ids) for c in res.completed)
    n_in = sum(len(r.prompt_ids) for r in reqs)
    return n_out / res.wall_s, n_in, n_out, res.wall_s, res.stats.steps


def random_prompts(n: int, length: int, vocab: int, seed: int):
    import torch
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (length,), generator=g).tolist() for _ in range(n)]


def time_decode_device(llm, cfg, batch: int, context: int, steps: int, warmup: int, tag: str):
    """Device time of `steps` decode steps at `batch` x `context`: (ms/step over the whole
    timed region, launches, per-step times).  One CUDA event after every step."""
    import torch

    from scratch_llm_b200.engine import RowInput
    from scratch_llm_b200.kernels import ops

    runner = llm.runner
    ids = [f"{tag}{i}" for i in range(batch)]
    prompts = random_prompts(batch, context, cfg.vocab_size, seed=batch)
    for rid, p in zip(ids, prompts):
        assert runner.admit(rid)
    for start in range(0, batch, 2):   # prefill two prompts per step
        runner.step([RowInput(rid, p) for rid, p in zip(ids[start:start + 2],
                                                        prompts[start:start + 2])])
    nxt = random_prompts(warmup + steps, batch, cfg.vocab_size, seed=99)
    out = torch.empty(batch, dtype=torch.int32, device=runner.device)
    scratch = torch.zeros(ops.argmax_scratch_bytes(batch), dtype=torch.uint8, device=runner.device)

    def one(k):
        logits = runner.step([RowInput(rid, [nxt[k][i]], [0]) for i, rid in enumerate(ids)])
        ops.argmax(logits, out, scratch, batch)   # greedy choice, as LLM.step does

    for k in range(warmup):
        one(k)
    torch.cuda.synchronize()
    before = ops.launch_count + runner.replayed_kernels
    marks = [torch.cuda.Event(enable_timing=True) for _ in range(steps + 1)]
    marks[0].record()
    for k in range(steps):
        one(warmup + k)
        marks[k + 1].record()
    torch.cuda.synchronize()
    launches = ops.launch_count + runner.replayed_kernels - before
    for rid in ids:
        runner.release(rid)
    ops.check_kernel_errors()
    per_step = [marks[k].elapsed_time(marks[k + 1]) for k in range(steps)]
    return marks[0].elapsed_time(marks[-1]) / steps, launches, per_step


def time_decode_e2e(llm, cfg, batch: int, context: int, steps: int, warmup: int):
    """Wall time of `steps` scheduler steps through LLM.submit/LLM.step: (ms/step, h2d, d2h)."""
    import torch

    from scratch_llm_b200 import Request, SamplingParams

    prompts = random_prompts(batch, context, cfg.vocab_size, seed=1000 + batch)
    # room for the steps in which later prompts are still read while earlier requests decode
    params = SamplingParams(temperature=0.0,
                            max_tokens=warmup + steps + 8 + batch + batch * context // 1024)
    for i, p in enumerate(prompts):
        llm.submit(Request(f"e{i}", p, params))
    produced = set()
    while len(produced) < batch:            # prompts are read; every request has a first token
        produced.update(llm.step())
    for _ in range(warmup):
        llm.step()
    stager = llm.runner._stager
    torch.cuda.synchronize()
    h0, d0 = stager.bytes_uploaded, llm.sampler.bytes_read
    t0 = time.perf_counter()
    n_tokens = 0
    for _ in range(steps):
        n_tokens += len(llm.step())
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    h2d = (stager.bytes_uploaded - h0) / steps
    d2h = (llm.sampler.bytes_read - d0) / steps
    llm.abort_all()
    assert n_tokens == batch * steps
    return wall * 1e3 / steps, h2d, d2h


def time_prefill(llm, cfg, tokens: int, reps: int = 9):
    """Times of `reps` prompt steps of `tokens` tokens (after three untimed ones), each from an
    empty cache."""
    import torch

    from scratch_llm_b200.engine import RowInput

    runner = llm.runner
    prompt = random_prompts(1, tokens, cfg.vocab_size, seed=7)[0]
    times = []
    for r in range(reps + 3):
        assert runner.admit("prefill")
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        runner.step([RowInput("prefill", prompt, [tokens - 1])])
        e1.record()
        torch.cuda.synchronize()
        if r >= 3:
            times.append(e0.elapsed_time(e1))
        runner.release("prefill")
    return times


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=10)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=SIZES["num_hidden_layers"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=1024)
    ap.add_argument("--prefill-tokens", type=int, default=2048)
    ap.add_argument("--page-size", type=int, default=64)
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 and 64 points")
    ap.add_argument("--sizes", default="llama-3-8b", choices=sorted(SIZES_BY_NAME),
                    help="layer sizes (the default is the configuration the metric is quoted on)")
    ap.add_argument("--serve", type=int, default=0, metavar="N",
                    help="also run the continuous-batching workload with N requests")
    ap.add_argument("--compare", default=None, choices=["nilevik", "vobosun", "titedra", "tubevik", "deganex",
                                                        "kumudra"],
                    help="instead of the headline workload: prefill and decode throughput of "
                         "this design beside the Llama-style model of equal size")
    ap.add_argument("--compare-sizes", default=None, choices=sorted(COMPARE_SIZES),
                    help="with --compare: one of the sizes (default: all)")
    args = ap.parse_args()
    if args.compare:
        if args.gpus != 1 or args.impl != "ours":
            print("--compare measures this engine on one GPU")
            return 2
        args.warmup = max(args.warmup, 3)
        return compare_main(args)
    sizes = SIZES_BY_NAME[args.sizes]
    if args.layers == SIZES["num_hidden_layers"] and args.sizes != "llama-3-8b":
        args.layers = sizes["num_hidden_layers"]
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this engine has no multi-GPU path (--gpus {args.gpus})")
        return 2
    args.warmup = max(args.warmup, 3)
    if args.impl == "reference":
        from baseline import reference_arm
        return reference_arm.main(args, sizes)

    import torch

    torch.cuda.set_device(0)
    pk = peaks()
    big = max(64, args.batch)
    capacity = big * (args.context + args.warmup + args.steps + 64) + 4096
    if args.serve:
        capacity = max(capacity, min(args.serve, 64) * 2600)
    cfg, model, llm, how = build_engine(args.layers, capacity, big + 1, args.page_size, sizes)

    with torch.no_grad():
        with ClockSampler(0) as clk_prefill:
            prefill_times = time_prefill(llm, cfg, args.prefill_tokens)
        with ClockSampler(0) as clk:
            ms, launches, per_step = time_decode_device(llm, cfg, args.batch, args.context,
                                                        args.steps, args.warmup, "d")
        with ClockSampler(0) as clk_e2e:
            e2e_ms, h2d, d2h = time_decode_e2e(llm, cfg, args.batch, args.context, args.steps,
                                               args.warmup)
        points = {}
        with ClockSampler(0) as clk_points:
            if not args.no_points:
                for b in (1, 64):
                    pms, _, _ = time_decode_device(llm, cfg, b, args.context,
                                                   max(8, args.steps // 2), args.warmup,
                                                   f"p{b}_")
                    points[f"decode_b{b}"] = round(b / pms * 1e3, 1)
        serve = None
        if args.serve:
            tok_s, n_in, n_out, seconds, steps = time_serve(llm, cfg, args.serve)
            serve = {"requests": args.serve, "generated_tok_s": round(tok_s, 1),
                     "prompt_tokens": n_in, "generated_tokens": n_out,
                     "seconds": round(seconds, 3), "steps": steps}

    prefill_ms = statistics.median(prefill_times)
    value = args.batch / ms * 1e3
    ctx_mid = args.context + args.warmup + args.steps / 2
    step_bytes = weight_bytes(sizes, args.layers) + \
        args.batch * ctx_mid * kv_bytes_per_token(sizes, args.layers)
    achieved = step_bytes / (ms * 1e-3) / 1e9
    flops = prefill_flops(sizes, args.layers, args.prefill_tokens)
    out = {
        "metric": f"decode tok/s at batch {args.batch} ({SIZE_LABELS[args.sizes]} sizes, "
                  "random weights)",
        "value": round(value, 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
        "warmup": args.warmup, "ms_per_step": round(ms, 4), "spread": spread(per_step),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic", "impl": "ours",
        "config": model_config(args.sizes, sizes, args.layers, args.batch, args.context,
                               args.prefill_tokens, pk["source"]),
        "engine": {"page_size": args.page_size, "weights_from": how},
        "e2e": {"value": round(args.batch / e2e_ms * 1e3, 1), "unit": "tok/s",
                "ms_per_step": round(e2e_ms, 4), "h2d_bytes_per_step": int(h2d),
                "d2h_bytes_per_step": int(d2h)},
        "gpu_launches": launches,
        "prefill": {"value": round(args.prefill_tokens / prefill_ms * 1e3, 1),
                    "tokens": args.prefill_tokens, "ms": round(prefill_ms, 3),
                    "frac": round(flops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4),
                    "spread": spread(prefill_times)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"],
                     "unit": "GB/s", "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
        "clocks": clk.summary,
        "clocks_regions": {"prefill": clk_prefill.summary, "e2e": clk_e2e.summary,
                           "points": clk_points.summary},
    }
    if serve is not None:
        out["serve"] = serve
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
