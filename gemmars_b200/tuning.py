"""Measurements that the dispatch rules rest on, to be run again on another GPU or another width.

    python -m gemmars_b200.tuning products [--shapes 4b,8b,32b] [--tokens 1,8,16,32,64]      (shapes: 0.6b 1.7b 4b 8b 14b 32b)
    python -m gemmars_b200.tuning timeline --shape 8b --batch 8 --context 8192 [--layers 6] [--prompt 2048]
                                           [--temperature 0.7]

``products``: every decode-shaped matrix product of a model shape (q/k/v, o, gate/up, down) with cold
weights, timed for every split of the inner dimension, beside the split ``kernels.gemm_tc_tiling``
picks by itself.  ``timeline``: the kernels of one replayed decode step (or, with ``--prompt``, of
one prompt step) as the device ran them, from CUPTI's kernel records: start, duration, and the gap
to the kernel before, which inside a replayed step is negative where dependent launch lets a kernel
start under its predecessor.  Both print plain text.
"""
from __future__ import annotations

import argparse
import re
import sys


def qwen3_shape(layers, hidden, heads, kv_heads, inter, tied):
    """A Qwen3 config.json object of the given layer sizes (heads of 128, the released vocabulary)."""
    return {"architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "num_hidden_layers": layers,
            "hidden_size": hidden, "num_attention_heads": heads, "num_key_value_heads": kv_heads, "head_dim": 128,
            "intermediate_size": inter, "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6,
            "attention_bias": False, "tie_word_embeddings": tied, "max_position_embeddings": 40960}


# The layer sizes of the released Qwen3 dense models; the dispatch rules were measured at 4b, 8b and 32b.
SHAPES = {
    "8b": ("Qwen3-8B shape", qwen3_shape(36, 4096, 32, 8, 12288, False)),
    "4b": ("Qwen3-4B shape", qwen3_shape(36, 2560, 32, 8, 9728, True)),
    "32b": ("Qwen3-32B shape", qwen3_shape(64, 5120, 64, 8, 25600, False)),
    "0.6b": ("Qwen3-0.6B shape", qwen3_shape(28, 1024, 16, 8, 3072, True)),
    "1.7b": ("Qwen3-1.7B shape", qwen3_shape(28, 2048, 16, 8, 6144, True)),
    "14b": ("Qwen3-14B shape", qwen3_shape(40, 5120, 40, 8, 17408, False)),
}


def toretar_shape(layers, width, heads, dim, rot_dim, vdim, rank, experts, top, ff, shared_ff, vocab=102400):
    """A Toretar config.json object of the given layer sizes (every layer alike)."""
    layer = {"type": "latent_attention",
             "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                       "scale": (dim + rot_dim) ** -0.5, "rot": {"base": 10000.0, "dims": rot_dim}},
             "mlp": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": 7.0},
                     "shared": {"ff": shared_ff, "limit": 7.0}}}
    return {"architecture": "Toretar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [layer] * layers}


def _pair(layers, width, heads, dim, rot_dim, vdim, rank, experts, top, ff, shared_ff, qwen_heads, qwen_kv):
    """A Toretar shape and the Qwen3 shape beside it: the same width, layers and vocabulary, heads
    of 128, and a feed-forward as wide as what one Toretar token runs (top experts + the shared one)."""
    q = qwen3_shape(layers, width, qwen_heads, qwen_kv, top * ff + shared_ff, False)
    q["vocab_size"] = 102400
    return toretar_shape(layers, width, heads, dim, rot_dim, vdim, rank, experts, top, ff, shared_ff), q


# Layer sizes in the range of released latent-attention mixture-of-experts models, four layers each
PAIRS = {
    "small": _pair(4, 1024, 8, 64, 32, 64, 256, 16, 2, 512, 1024, 8, 4),
    "lite": _pair(4, 2048, 16, 128, 64, 128, 512, 64, 6, 1408, 2816, 16, 8),
    "mid": _pair(4, 4096, 32, 128, 64, 128, 512, 32, 4, 2048, 4096, 32, 8),
}


# the same pairs by name, for ``timeline --shape toretar-lite`` and ``--shape beside-lite``
PAIR_SHAPES = {}
for _name, (_t, _q) in PAIRS.items():
    PAIR_SHAPES[f"toretar-{_name}"] = (f"Toretar shape '{_name}'", _t)
    PAIR_SHAPES[f"beside-{_name}"] = (f"Qwen3 shape beside Toretar '{_name}'", _q)


def kuporax_shape(width, ff, heads, window, order=("delta", "parallel", "parallel", "delta"), vocab=102400, positions=16384):
    """A Kuporax config.json object with ``heads`` heads of 128 in every mixer: delta layers with
    half as many q/k heads as heads; side-by-side layers of windowed attention (keys and values of
    128, a quarter as many kv heads) and a state-space branch with twice as many heads of 64 and a
    state of 128."""
    delta = {"type": "delta", "mixer": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "conv": 4},
             "mlp": {"kind": "dense", "ff": ff}}
    parallel = {"type": "parallel",
                "mixer": {"left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "conv": 3,
                                   "scale": 128 ** -0.5, "softcap": 30.0, "mask": {"size": window},
                                   "rot": {"base": 1000000.0, "dims": 128}},
                          "right": {"heads": 2 * heads, "vdim": 64, "state": 128, "groups": max(1, heads // 4),
                                    "norm_groups": max(1, heads // 4), "conv": 4},
                          "left_scale": 1.0, "right_scale": 1.0},
                "mlp": {"kind": "dense", "ff": ff}}
    return {"architecture": "Kuporax", "vocab": vocab, "width": width, "max_positions": positions, "logit_scale": 1.0,
            "norm": {"eps": 1e-6}, "layers": [delta if kind == "delta" else parallel for kind in order]}


def _kuporax_pair(width, ff, heads, window):
    """A Kuporax shape and the Qwen3 shape beside it: the same width, depth, vocabulary and
    feed-forward, heads of 128 with a quarter as many kv heads, and the same window on every layer."""
    k = kuporax_shape(width, ff, heads, window)
    q = qwen3_shape(len(k["layers"]), width, heads, max(1, heads // 4), ff, False)
    q.update({"vocab_size": k["vocab"], "use_sliding_window": True, "sliding_window": window,
              "layer_types": ["sliding_attention"] * len(k["layers"])})
    return k, q


# Layer sizes in the range of released models that mix recurrent layers with windowed attention, four layers each
KUPORAX_PAIRS = {
    "small": _kuporax_pair(1024, 4096, 8, 512),
    "lite": _kuporax_pair(2048, 8192, 16, 1024),
    "mid": _kuporax_pair(4096, 12288, 32, 2048),
}
for _name, (_k, _q) in KUPORAX_PAIRS.items():
    PAIR_SHAPES[f"kuporax-{_name}"] = (f"Kuporax shape '{_name}'", _k)
    PAIR_SHAPES[f"beside-kuporax-{_name}"] = (f"Qwen3 shape beside Kuporax '{_name}'", _q)


def dalerax_shape(width, ff, heads, window, experts, top, order=("wkv", "attention", "attention", "wkv"),
                  vocab=102400, positions=16384):
    """A Dalerax config.json object: attention layers of ``heads`` heads of 128 (a quarter as many
    kv heads, four kept first tokens, a sink, stretched long wavelengths), the second of which reads
    the first one's keys and values; recurrent layers of heads of 64 over the whole width with a
    decay of rank 64.  The first layer's feed-forward is dense; the others route ``top`` of
    ``experts`` experts beside a shared one, sized so that a token passes ``ff`` hidden units in all."""
    shared_ff = ff // 4
    expert_ff = (ff - shared_ff) // top
    rot = {"base": 1000000.0, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    layers, first_attention = [], None
    for i, kind in enumerate(order):
        if kind == "wkv":
            mixer = {"heads": width // 64, "dim": 64, "rank": 64}
        else:
            mixer = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "mask": {"size": window, "keep_first": 4}, "rot": rot}
            if first_attention is None:
                first_attention = i
            else:
                mixer["kv_from"] = first_attention
        mlp = ({"kind": "dense", "ff": ff} if i == 0 else
               {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": expert_ff}, "shared": {"ff": shared_ff}})
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Dalerax", "vocab": vocab, "width": width, "max_positions": positions, "logit_scale": 1.0,
            "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "layers": layers}


# Dalerax beside Kuporax, the nearest design the package has (recurrent layers around windowed
# attention): the same width, depth, vocabulary, heads, window and hidden units a token passes
DALERAX_PAIRS = {
    "small": (dalerax_shape(1024, 4096, 8, 512, 16, 3), kuporax_shape(1024, 4096, 8, 512)),
    "lite": (dalerax_shape(2048, 8192, 16, 1024, 32, 6), kuporax_shape(2048, 8192, 16, 1024)),
    "mid": (dalerax_shape(4096, 12288, 32, 2048, 32, 6), kuporax_shape(4096, 12288, 32, 2048)),
}
for _name, (_d, _k) in DALERAX_PAIRS.items():
    PAIR_SHAPES[f"dalerax-{_name}"] = (f"Dalerax shape '{_name}'", _d)


def nogosun_shape(width, ff, heads, window, experts, top, order=("channel_delta", "parallel", "attention", "attention"),
                  vocab=102400):
    """A Nogosun config.json object: attention layers of ``heads`` heads of 128 whose values are their
    keys (a quarter as many kv heads, four kept first tokens, half of every head rotated with
    scaling), the second of which runs the first one's tensors again; a delta rule with a decay per
    key channel, ``heads`` heads of 128 over half as many q/k heads, a filter of 4 taps, inner sizes
    of 64; a two-branch layer of tempered attention (half the heads, over every key) beside gated
    linear attention (half the heads, keys of 64 and values of 128).  Every layer routes ``top`` of
    ``experts`` experts without gates, sized so that a token passes ``ff`` hidden units in all."""
    rot = {"base": 1000000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 8192, "fast": 16.0, "slow": 2.0}}
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff // top}}
    half = max(1, heads // 2)
    mixers = {
        "channel_delta": {"heads": heads, "kv_heads": half, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 64, "gate_rank": 64},
        "parallel": {"left": {"heads": half, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                              "softcap": 30.0, "q_temp": {"coef": 0.25, "every": 512}},
                     "right": {"heads": half, "dim": 64, "vdim": 128, "tau": 8.0, "rank": 64},
                     "left_scale": 1.0, "right_scale": 1.0},
        "attention": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                      "mask": {"size": window, "keep_first": 4}, "rot": rot},
    }
    layers, first = [], {}
    for i, kind in enumerate(order):
        layer = {"type": kind, "mixer": mixers[kind], "mlp": mlp}
        if kind == "attention" and kind in first:
            layer["weights_of"] = first[kind]
        first.setdefault(kind, i)
        layers.append(layer)
    return {"architecture": "Nogosun", "vocab": vocab, "width": width, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "layers": layers}


# Nogosun beside Dalerax, the nearest design the package has (parallel blocks, kept first tokens beside a
# window, a recurrence with a decay per key channel, routed experts): the same width, depth,
# vocabulary, heads, window, experts and hidden units a token passes
NOGOSUN_PAIRS = {
    "small": (nogosun_shape(1024, 4096, 8, 512, 16, 4), dalerax_shape(1024, 4096, 8, 512, 16, 3)),
    "lite": (nogosun_shape(2048, 8192, 16, 1024, 32, 4), dalerax_shape(2048, 8192, 16, 1024, 32, 6)),
    "mid": (nogosun_shape(4096, 12288, 32, 2048, 32, 4), dalerax_shape(4096, 12288, 32, 2048, 32, 6)),
}
for _name, (_n, _d) in NOGOSUN_PAIRS.items():
    PAIR_SHAPES[f"nogosun-{_name}"] = (f"Nogosun shape '{_name}'", _n)


def mevuvik_shape(width, ff, heads, rank, q_rank, experts, top, vocab=102400):
    """A Mevuvik config.json object of three layers, the second run twice: a two-branch layer of
    attention without positions (half of ``heads`` heads of 128, an eighth as many kv heads as heads)
    beside matrix memory (as many heads, keys of 64 and values of 128), experts behind it; a latent
    attention layer of ``heads`` heads of 128 + 64 with values of 128, experts behind it; a two-branch
    layer again, a dense feed-forward behind it.  A token passes ``ff`` hidden units in every layer."""
    half = max(1, heads // 2)
    moe = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": 2.0}, "expert": {"ff": ff // top}}
    pair = {"left": {"heads": half, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "scale": 128 ** -0.5},
            "right": {"heads": half, "dim": 64, "vdim": 128, "gate_cap": 12.0}, "left_scale": 1.0, "right_scale": 1.0}
    latent = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": q_rank, "kv_rank": rank, "scale": 192 ** -0.5,
              "rot": {"base": 1000000.0, "dims": 64}}
    return {"architecture": "Mevuvik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
            "logit_softcap": 30.0, "loop": {"start": 1, "stop": 2, "times": 2},
            "layers": [{"type": "parallel", "mixer": pair, "mlp": moe},
                       {"type": "latent_attention", "mixer": latent, "mlp": moe},
                       {"type": "parallel", "mixer": pair, "mlp": {"kind": "dense", "ff": ff}}]}


# Mevuvik beside Nogosun, the nearest design the package has (attention over every key beside a linear
# recurrence, experts without gates, layers that run again): the same width, runs of layers, vocabulary,
# heads, experts and hidden units a token passes.  Its latent attention's like is Toretar's ("toretar-*").
MEVUVIK_PAIRS = {
    "small": (mevuvik_shape(1024, 4096, 8, 256, 512, 16, 4), nogosun_shape(1024, 4096, 8, 512, 16, 4)),
    "lite": (mevuvik_shape(2048, 8192, 16, 512, 1024, 32, 4), nogosun_shape(2048, 8192, 16, 1024, 32, 4)),
    "mid": (mevuvik_shape(4096, 12288, 32, 512, 1536, 32, 4), nogosun_shape(4096, 12288, 32, 2048, 32, 4)),
}
for _name, (_m, _n) in MEVUVIK_PAIRS.items():
    PAIR_SHAPES[f"mevuvik-{_name}"] = (f"Mevuvik shape '{_name}'", _m)


def fezozen_shape(width, ff, heads, window, rank, experts, top, order=("attention_2", "attention", "latent_attention", "attention_2"),
                  vocab=102400):
    """A Fezozen config.json object: attention over every key (``heads`` heads of 128, a quarter as many
    kv heads, half of every head turned with scaling, capped scores), windowed attention with unit q and
    k (the same heads, every dim turned), the second of which runs the first one's tensors again, and
    windowed latent attention (``heads`` heads of 128 + 64 with values of 128).  Every layer routes
    ``top`` of ``experts`` gated experts, sized so that a token passes ``ff`` hidden units in all."""
    heads_128 = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    stretched = {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}
    mixers = {
        "attention": {**heads_128, "softcap": 30.0, "rot": {"base": 1000000.0, "dims": 64, "scaling": stretched}},
        "attention_2": {**heads_128, "mask": {"size": window}, "rot": {"base": 1000000.0, "dims": 128}},
        "latent_attention": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": rank, "scale": 192 ** -0.5,
                             "mask": {"size": window}, "rot": {"base": 1000000.0, "dims": 64, "scaling": stretched}},
    }
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff // top}}
    layers, first = [], {}
    for i, kind in enumerate(order):
        layer = {"type": kind, "mixer": mixers[kind], "mlp": mlp}
        if kind in first:
            layer["weights_of"] = first[kind]
        first.setdefault(kind, i)
        layers.append(layer)
    return {"architecture": "Fezozen", "vocab": vocab, "width": width, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "layers": layers}


# Fezozen beside Toretar, the nearest design the package has (softmax attention alone, pairs turned side by
# side, latent attention with a gate, gated experts): the same width, layers, vocabulary, heads, latent and
# hidden units a token passes (Toretar's through one expert fewer and a shared expert as wide as one).  Its
# grouped-query attention's like is the capped attention of Nogosun ("nogosun-*").
def _fezozen_pair(width, ff, heads, window, rank, experts, top):
    return (fezozen_shape(width, ff, heads, window, rank, experts, top),
            toretar_shape(4, width, heads, 128, 64, 128, rank, experts, top - 1, ff // top, ff // top))


FEZOZEN_PAIRS = {
    "small": _fezozen_pair(1024, 4096, 8, 512, 256, 16, 4),
    "lite": _fezozen_pair(2048, 8192, 16, 1024, 512, 32, 4),
    "mid": _fezozen_pair(4096, 12288, 32, 2048, 512, 32, 4),
}
for _name, (_f, _t) in FEZOZEN_PAIRS.items():
    PAIR_SHAPES[f"fezozen-{_name}"] = (f"Fezozen shape '{_name}'", _f)
    PAIR_SHAPES[f"beside-fezozen-{_name}"] = (f"Toretar shape beside Fezozen '{_name}'", _t)


def random_engine(cfg, max_batch, cache_tokens, options=""):
    """An engine over random weights of ``cfg`` made on the device; the tensors are taken out of
    their dict as they are bound, so that a model of 65 GB and its stacked q/k/v and gate/up copies
    never sit in memory side by side."""
    import torch
    from .engine.engine import Engine, EngineOptions
    from .weights.random_init import random_weights
    torch.cuda.set_device(0)
    tensors = random_weights(cfg, seed=0, device="cuda:0")
    opts = EngineOptions.parse({"dtype": "bfloat16", "max_batch": str(max_batch), "max_tokens": str(cache_tokens),
                                "prefill_chunk": "2048"})
    for pair in filter(None, (p.strip() for p in options.split(";"))):
        opts.set(*[x.strip() for x in pair.split("=", 1)])
    return Engine.from_config(cfg, tensors, opts, consume=True)


def synthetic_fill(runner, slots, length):
    """Brings every slot to ``length`` cached tokens by reserving the pages and writing random
    keys and values (what a timing needs of a cache, without running prompts)."""
    for s in slots:
        runner.cache.extend(s, length)
    runner.cache.sync()
    for g in runner.cache.kv_groups:
        for t in (g.k, g.v):
            for layer in range(t.shape[0]):
                t[layer].normal_(0.0, 1.0)


# ---------------------------------------------------------------------------------------- products

def sweep_products(shapes, tokens, hbm_gbs=6542.0, out=sys.stdout):
    import torch
    from . import kernels
    torch.manual_seed(0)
    for name in shapes:
        cfg = SHAPES[name][1]
        h, hd = cfg["hidden_size"], cfg["head_dim"]
        qkv = (cfg["num_attention_heads"] + 2 * cfg["num_key_value_heads"]) * hd
        ao, inter = cfg["num_attention_heads"] * hd, cfg["intermediate_size"]
        products = [("qkv", qkv, h, "bf16"), ("o", h, ao, "acc"), ("gate_up", inter, h, "gated"), ("down", h, inter, "acc")]
        for m in tokens:
            for what, n, k, mode in products:
                rows = 2 * n if mode == "gated" else n
                copies = max(2, int(1.0e9 // (rows * k * 2)))          # more weights than L2 holds: every launch reads cold
                ws = [torch.randn(rows, k, device="cuda").bfloat16() for _ in range(copies)]
                x = torch.randn(m, k, device="cuda").bfloat16()
                y = torch.zeros(m, n, device="cuda", dtype=torch.float32 if mode == "acc" else torch.bfloat16)
                auto = kernels.gemm_tc_tiling(m, n, k, gated=(mode == "gated"))
                res = []
                for splits in (1, 2, 4, 8):
                    if k // 64 // splits < 2:
                        continue

                    def run():
                        for w in ws:
                            kernels.gemm_tc(x, w, y, accumulate=(mode == "acc"), splits=splits, swiglu=(mode == "gated"))
                    run()
                    torch.cuda.synchronize()
                    g = torch.cuda.CUDAGraph()
                    with torch.cuda.graph(g):
                        run()
                    g.replay()
                    torch.cuda.synchronize()
                    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                    e0.record()
                    for _ in range(5):
                        g.replay()
                    e1.record()
                    torch.cuda.synchronize()
                    res.append((e0.elapsed_time(e1) * 1e3 / 5 / copies, splits))
                best = min(res)
                ideal = rows * k * 2 / hbm_gbs / 1e3
                chosen = dict((sp, us) for us, sp in res).get(auto[1], float("nan"))
                print(f"{name:3s} {m:3d} tokens {what:8s} {rows:6d} x {k:5d}  bytes take {ideal:6.1f} us | "
                      + " ".join(f"x{sp}: {us:6.1f}" for us, sp in res)
                      + f" | best x{best[1]} {best[0]:6.1f} us | chosen x{auto[1]} (tile {auto[0]}) {chosen:6.1f} us", file=out, flush=True)
                del ws
    kernels.check_status()


# ---------------------------------------------------------------------------------------- timeline

def _short(name: str) -> str:
    name = name.replace("void ", "").replace("(anonymous namespace)::", "").replace("<unnamed>::", "")
    m = re.match(r"([A-Za-z0-9_]+)(<[^>]*>)?", name)
    return ((m.group(1) + (m.group(2) or "")) if m else name)[:46]


def timeline(shape, batch, context, layers, prompt, temperature, out=sys.stdout):
    import torch
    from torch.profiler import ProfilerActivity, profile
    from .engine.step import StepItem
    from .sampling.sampler import BatchSampler, SamplingParams
    label, cfg = {**SHAPES, **PAIR_SHAPES}[shape]
    if "layers" in cfg:
        if not cfg.get("loop"):           # a loop's layers are counted by their runs and kept whole
            cfg = dict(cfg, layers=cfg["layers"][:layers or len(cfg["layers"])])
        n_layers, vocab = len(cfg["layers"]), cfg["vocab"]
    else:
        cfg = dict(cfg, num_hidden_layers=layers or cfg["num_hidden_layers"])
        n_layers, vocab = cfg["num_hidden_layers"], cfg["vocab_size"]
    eng = random_engine(cfg, max(batch, 1), max(batch, 1) * (max(context, prompt) + 128))
    runner = eng.runner
    if prompt:
        toks = torch.randint(0, vocab, (prompt,), generator=torch.Generator().manual_seed(3)).tolist()

        def step():
            s = runner.open()
            runner.step([StepItem(s, toks, [prompt - 1])])
            torch.cuda.synchronize()
            runner.close(s)
        what = f"prompt of {prompt} tokens"
    else:
        slots = [runner.open() for _ in range(batch)]
        synthetic_fill(runner, slots, context - 50)
        sampler = BatchSampler([SamplingParams(temperature=temperature)] * batch, runner.device)
        rows = list(range(batch))
        state = {"logits": runner.step([StepItem(s, [5], [0]) for s in slots])}

        def step():
            # as the generation loop steps: draw, launch the next step from the drawn tokens where
            # they lie, then read them on the host
            drawn = sampler.draw(state["logits"], rows)
            nxt = runner.decode_from_device(slots, drawn) if eng.options.decode_ahead else None
            toks = sampler.read(drawn)
            state["logits"] = nxt if nxt is not None else runner.step([StepItem(s, [t], [0]) for s, t in zip(slots, toks)])
        what = f"decode step, batch {batch}, context {context}" + (f", temperature {temperature}" if temperature > 0 else "")
    for _ in range(5):
        step()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(8):
        step()
    e1.record()
    torch.cuda.synchronize()
    print(f"{label}, {n_layers} layers, {what}: {e0.elapsed_time(e1) / 8 * 1e3:.1f} us a step "
          "(CUDA events, host turnaround included)", file=out)
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(3):
            step()
        torch.cuda.synchronize()
    ev = [e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA and "Memset" not in e.name]
    ev.sort(key=lambda e: e.time_range.start)
    last = ev[-(len(ev) // 3):]
    t0, prev_end, rows = last[0].time_range.start, last[0].time_range.start, []
    for e in last:
        rows.append((_short(e.name), e.time_range.start - t0, e.time_range.end - e.time_range.start,
                     e.time_range.start - prev_end))
        prev_end = max(prev_end, e.time_range.end)
    print(f"{len(rows)} kernels and copies in the step, {last[-1].time_range.end - t0:.1f} us from the first start to the last end", file=out)
    mid = len(rows) // 2
    print("-- the middle of the step (us: start, duration, gap to the end of everything before)", file=out)
    for name, s, d, gap in rows[max(0, mid - 6): mid + 12]:
        print(f"{name:46s} {s:9.1f} {d:8.1f} {gap:7.1f}", file=out)
    print("-- the end of the step", file=out)
    for name, s, d, gap in rows[-8:]:
        print(f"{name:46s} {s:9.1f} {d:8.1f} {gap:7.1f}", file=out)
    print("-- per kernel (calls, sum and mean of durations, sum of gaps)", file=out)
    tot = {}
    for name, s, d, gap in rows:
        a = tot.setdefault(name, [0, 0.0, 0.0])
        a[0] += 1
        a[1] += d
        a[2] += gap
    for k, (n, d, g) in sorted(tot.items(), key=lambda kv: -kv[1][1]):
        print(f"{k:46s} {n:4d} {d:9.1f} {d / n:8.1f} {g:8.1f}", file=out)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m gemmars_b200.tuning", description=__doc__.split("\n\n")[0])
    sub = ap.add_subparsers(dest="command", required=True)
    p = sub.add_parser("products", help="decode-shaped products at every split, with cold weights")
    p.add_argument("--shapes", default="4b,8b,32b")
    p.add_argument("--tokens", default="1,8,16,32,64")
    t = sub.add_parser("timeline", help="the kernels of one replayed decode step or one prompt step")
    t.add_argument("--shape", default="8b", choices=sorted(SHAPES) + sorted(PAIR_SHAPES))
    t.add_argument("--batch", type=int, default=8)
    t.add_argument("--context", type=int, default=8192)
    t.add_argument("--layers", type=int, default=6, help="layers of the model that is built (0: all)")
    t.add_argument("--prompt", type=int, default=0, help="time a prompt of this many tokens instead of a decode step")
    t.add_argument("--temperature", type=float, default=0.0)
    args = ap.parse_args(argv)
    if args.command == "products":
        sweep_products([s.strip() for s in args.shapes.split(",")], [int(x) for x in args.tokens.split(",")])
    else:
        timeline(args.shape, args.batch, args.context, args.layers, args.prompt, args.temperature)
    return 0


if __name__ == "__main__":
    sys.exit(main())
