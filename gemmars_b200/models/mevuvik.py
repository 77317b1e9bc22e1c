"""Mevuvik: configuration, plan, tensor names.

A pre-norm decoder whose norms have one number for all coordinates:
x += m * ls1 * mixer(norm1(x)), then x += m * ls2 * ffn(norm2(x)), with m the configuration's
``residual_mult`` and ls1, ls2 factors per feature.  The token's embedding passes a norm before it
becomes the stream; the logits are capped.  Layers ``loop.start`` .. ``loop.stop`` - 1 run
``loop.times`` times in a row with the same tensors, each pass with caches and states of its own, and
before pass t row t of ``loop.step`` is added to the stream.  Two mixers:

* ``latent_attention``: queries, and keys with values, each through a normed latent; the last
  ``rot_dim`` query/key dims of a head are rotated in the half layout, their key part shared by all heads.
* ``parallel``: two mixers on the same input, each times a factor: ``left``, grouped-query softmax
  attention without positions, with one sigmoid gate per head; ``right``, matrix memory with
  exponential gates (an mLSTM).

The feed-forward is down relu(up h)^2, or routes every token to ``top`` of ``experts`` such small layers
by sigmoid scores with a correction that only the choice sees; or there is none (``mlp: null``).

config.json::

    {"architecture": "Mevuvik", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "logit_softcap": null | c, "loop": null | {"start", "stop", "times"},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}},
                 "mlp": null | {"kind": "dense", "ff"}},
                {"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale"},
                           "right": {"heads", "dim", "vdim", "gate_cap"}, "left_scale", "right_scale"},
                 "mlp": null | {"kind": "moe", "router": {"experts", "top", "scale"}, "expert": {"ff"}}}, ...]}

Tensors: ``embed``, ``embed.norm``, ``loop.step``, ``l<i>.{norm1,norm2,ls1,ls2}``, ``final.norm``, ``head``;
``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}`` (latent_attention); ``l<i>.mix.left.{q,k,v,g,o}`` and
``l<i>.mix.right.{q,k,v,g,i,i.b,f,f.b,norm,o}`` (parallel); ``l<i>.mlp.{up,down}`` or
``l<i>.mlp.{router,correction,e<j>.up,e<j>.down}``.

This module is all that knows the architecture: it turns the configuration into a ``ModelPlan`` of
generic parts (``prenorm`` block with ``channel_scale``, ``latent_attention``, ``capped_attention``,
``matrix_memory``, ``side_by_side``, ``plain_mlp``, ``moe`` without gates, ``rmsnorm``, ``rotary``, ``add_row``).
"""
from __future__ import annotations

import dataclasses
from typing import Optional, Tuple

from ..config.base import ConfigError, ModelConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

MIXERS = ("latent_attention", "parallel")
FFN_KINDS = ("dense", "moe")


def _num(problems, where, obj, name, kind=int, allow_zero=False, optional=False, signed=False):
    v = obj.get(name) if isinstance(obj, dict) else None
    if v is None and optional:
        return None
    if kind is int and isinstance(v, float) and v.is_integer():
        v = int(v)                                   # a count written as 256.0
    ok = isinstance(v, int) and not isinstance(v, bool) if kind is int else (
        isinstance(v, (int, float)) and not isinstance(v, bool))
    if not ok:
        problems.append(f"{where}.{name}: expected {'an integer' if kind is int else 'a number'}, got {v!r}")
        return None
    if not signed and (v < 0 or (v == 0 and not allow_zero)):
        problems.append(f"{where}.{name}: must be positive, got {v!r}")
        return None
    return kind(v)


def _check_latent(p, w, m):
    for name in ("heads", "vdim", "q_rank", "kv_rank"):
        _num(p, w, m, name)
    dim = _num(p, w, m, "dim", allow_zero=True)
    rd = _num(p, w, m, "rot_dim", allow_zero=True)
    _num(p, w, m, "scale", float, signed=True)
    if dim == 0 and rd == 0:
        p.append(f"{w}: dim and rot_dim are both 0")
    if rd:
        rot = m.get("rot")
        _num(p, w + ".rot", rot, "base", float)
        dims = _num(p, w + ".rot", rot, "dims", allow_zero=True)
        if dims is not None and (dims % 2 or dims > rd):
            p.append(f"{w}.rot.dims: {dims} is odd or more than rot_dim ({rd})")


def _check_parallel(p, w, m):
    left, right = m.get("left"), m.get("right")
    if not isinstance(left, dict) or not isinstance(right, dict):
        p.append(f"{w}: expected the objects left and right")
        return
    heads, g = _num(p, w + ".left", left, "heads"), _num(p, w + ".left", left, "kv_heads")
    if heads and g and heads % g:
        p.append(f"{w}.left: {heads} heads are not a multiple of {g} kv_heads")
    for name in ("dim", "vdim"):
        _num(p, w + ".left", left, name)
        _num(p, w + ".right", right, name)
    _num(p, w + ".left", left, "scale", float, signed=True)
    _num(p, w + ".right", right, "heads")
    _num(p, w + ".right", right, "gate_cap", float)
    _num(p, w, m, "left_scale", float, signed=True)
    _num(p, w, m, "right_scale", float, signed=True)


def _check_mlp(p, w, mlp):
    kind = mlp.get("kind") if isinstance(mlp, dict) else mlp
    if kind not in FFN_KINDS:
        p.append(f"{w}.kind: unknown feed-forward {kind!r} (known: {', '.join(FFN_KINDS)})")
    elif kind == "dense":
        _num(p, w, mlp, "ff")
    else:
        router = mlp.get("router")
        experts, top = _num(p, w + ".router", router, "experts"), _num(p, w + ".router", router, "top")
        if experts and top and top > experts:
            p.append(f"{w}.router.top: {top} of {experts} experts")
        _num(p, w + ".router", router, "scale", float, signed=True)
        _num(p, w + ".expert", mlp.get("expert"), "ff")


@dataclasses.dataclass(frozen=True)
class MevuvikConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    #: (start, stop, times), or None: no layer runs more than once
    loop: Optional[Tuple[int, int, int]]
    #: one entry per layer, as config.json lists them (checked; plain dicts)
    layers: Tuple[dict, ...]

    @classmethod
    def from_dict(cls, raw):
        if not isinstance(raw, dict):
            raise ConfigError("config.json: the top level must be an object")
        p = []
        vocab = _num(p, "config", raw, "vocab")
        width = _num(p, "config", raw, "width")
        eps = _num(p, "norm", raw.get("norm"), "eps", float, allow_zero=True)
        mult = _num(p, "config", raw, "residual_mult", float, signed=True)
        cap = _num(p, "config", raw, "logit_softcap", float, allow_zero=True, optional=True)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            p.append("layers: expected a list of at least one layer")
            layers = []
        for i, layer in enumerate(layers):
            w = f"layers[{i}]"
            if not isinstance(layer, dict):
                p.append(f"{w}: expected an object")
                continue
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in MIXERS:
                p.append(f"{w}.type: unknown mixer {kind!r} (known: {', '.join(MIXERS)})")
                continue
            if not isinstance(m, dict):
                p.append(f"{w}.mixer: expected an object")
                continue
            (_check_latent if kind == "latent_attention" else _check_parallel)(p, w + ".mixer", m)
            if layer.get("mlp") is not None:
                _check_mlp(p, w + ".mlp", layer["mlp"])
        loop = None
        if raw.get("loop") is not None:
            start = _num(p, "loop", raw["loop"], "start", allow_zero=True)
            stop = _num(p, "loop", raw["loop"], "stop")
            times = _num(p, "loop", raw["loop"], "times")
            if None not in (start, stop, times):
                if not start < stop <= len(layers):
                    p.append(f"loop: layers {start} to {stop} of {len(layers)} are no range")
                loop = (start, stop, times)
        if p:
            raise ConfigError("config.json: " + "; ".join(p))
        return cls(vocab=vocab, width=width, norm_eps=eps, residual_mult=mult, logit_softcap=cap or None, loop=loop,
                   layers=tuple(layers))

    def to_dict(self):
        loop = None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop))
        return {"architecture": "Mevuvik", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap, "loop": loop,
                "layers": [dict(layer) for layer in self.layers]}


def _latent_spec(cfg, m, prefix) -> PartSpec:
    rd, rot = int(m["rot_dim"]), m.get("rot") or {}
    position = None
    if rd and int(rot.get("dims", 0)):
        position = PartSpec("rotary", {"head_dim": rd, "rotary_dim": int(rot["dims"]), "theta": float(rot["base"]),
                                       "layout": "half"})
    names = {k: prefix + k for k in ("dq", "uq", "dkv", "uk", "uv", "o")}
    names.update({"dq_norm": prefix + "dq.norm", "dkv_norm": prefix + "dkv.norm"})
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": rd, "vdim": int(m["vdim"]),
        "rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]), "scale": float(m["scale"]), "norm_eps": cfg.norm_eps,
        "gate": False, "window": None, "position": position}, names)


def _parallel_spec(cfg, m, prefix) -> PartSpec:
    left, right = m["left"], m["right"]
    lspec = PartSpec("capped_attention", {
        "hidden_size": cfg.width, "heads": int(left["heads"]), "kv_heads": int(left["kv_heads"]), "dim": int(left["dim"]),
        "vdim": int(left["vdim"]), "scale": float(left["scale"]), "window": None, "gate": "head", "position": None},
        {k: f"{prefix}left.{k}" for k in ("q", "k", "v", "g", "o")})
    rnames = {k: f"{prefix}right.{k}" for k in ("q", "k", "v", "g", "i", "f", "norm", "o")}
    rnames.update({"i_bias": prefix + "right.i.b", "f_bias": prefix + "right.f.b"})
    rspec = PartSpec("matrix_memory", {
        "hidden_size": cfg.width, "heads": int(right["heads"]), "dim": int(right["dim"]), "vdim": int(right["vdim"]),
        "gate_cap": float(right["gate_cap"]), "norm_eps": cfg.norm_eps}, rnames)
    return PartSpec("side_by_side", {"branches": [{"name": "left", "spec": lspec, "scale": float(m["left_scale"])},
                                                  {"name": "right", "spec": rspec, "scale": float(m["right_scale"])}]})


def _ffn_spec(cfg, mlp, prefix) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("plain_mlp", {"hidden_size": cfg.width, "intermediate_size": int(mlp["ff"]), "activation": "relu2"},
                        {"up": prefix + "up", "down": prefix + "down"})
    router = mlp["router"]
    experts = int(router["experts"])
    names = {"router": prefix + "router", "router_bias": prefix + "correction"}
    for e in range(experts):
        names[f"e{e}.up"], names[f"e{e}.down"] = f"{prefix}e{e}.up", f"{prefix}e{e}.down"
    return PartSpec("moe", {"hidden_size": cfg.width, "experts": experts, "top": int(router["top"]),
                            "ff": int(mlp["expert"]["ff"]), "limit": None, "router_bias": True, "gated": False,
                            "activation": "relu2", "routing": "sigmoid", "routing_scale": float(router["scale"]),
                            "shared": None}, names)


def runs(cfg: MevuvikConfig) -> list:
    """[(layer, number of the loop's pass that starts with this run, or None)] in the order of the runs."""
    n = len(cfg.layers)
    if cfg.loop is None:
        return [(i, None) for i in range(n)]
    start, stop, times = cfg.loop
    passes = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    return [(i, None) for i in range(start)] + passes + [(i, None) for i in range(stop, n)]


def build_plan(cfg: MevuvikConfig, names=None) -> ModelPlan:
    def norm(name):
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "scalar": True}, {"weight": name})

    def scale(name):
        return PartSpec("channel_scale", {"size": cfg.width, "factor": cfg.residual_mult}, {"weight": name})

    layers, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        m, prefix = layer["mixer"], f"l{i}.mix."
        mixer = _latent_spec(cfg, m, prefix) if layer["type"] == "latent_attention" else _parallel_spec(cfg, m, prefix)
        parts = {"mixer_norm": norm(f"l{i}.norm1"), "mixer": mixer, "mixer_scale": scale(f"l{i}.ls1")}
        if layer.get("mlp") is not None:
            parts.update({"ffn_norm": norm(f"l{i}.norm2"), "ffn": _ffn_spec(cfg, layer["mlp"], f"l{i}.mlp."),
                          "ffn_scale": scale(f"l{i}.ls2")})
        else:
            ignored += [f"l{i}.norm2", f"l{i}.ls2"]          # a layer without feed-forward has no use for them
        layers.append(LayerSpec(parts, "prenorm"))

    def step(t):
        if t is None:
            return None
        return PartSpec("add_row", {"size": cfg.width, "rows": cfg.loop[2], "row": t}, {"weight": "loop.step"})

    plan = ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": None,
                                         "norm": {"eps": cfg.norm_eps, "scalar": True}},
                           {"weight": "embed", "norm": "embed.norm"}),
        layers=layers, schedule=[ScheduleEntry(i, before=step(t)) for i, t in runs(cfg)], final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "logit_softcap": cfg.logit_softcap},
                      {"weight": "head"}),
        max_positions=0, stop_ids=[], ignored_tensors=ignored)
    plan.validate()
    return plan


def checkpoint_layout(cfg: MevuvikConfig) -> dict:
    """{tensor name: (shape, kind)} of a complete checkpoint (kind as weights.random_init reads it)."""
    w = cfg.width
    out = {"embed": ((cfg.vocab, w), "matrix"), "embed.norm": ((), "norm")}
    if cfg.loop is not None:
        out["loop.step"] = ((cfg.loop[2], w), "small")
    for i, layer in enumerate(cfg.layers):
        m, p = layer["mixer"], f"l{i}.mix."
        out.update({f"l{i}.norm1": ((), "norm"), f"l{i}.ls1": ((w,), "norm")})
        if layer["type"] == "latent_attention":
            nh, d, rd, vd, rq, r = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            out.update({p + "dq": ((rq, w), "matrix"), p + "dq.norm": ((rq,), "norm"), p + "uq": ((nh * (d + rd), rq), "matrix"),
                        p + "dkv": ((r + rd, w), "matrix"), p + "dkv.norm": ((r,), "norm"), p + "uk": ((nh * d, r), "matrix"),
                        p + "uv": ((nh * vd, r), "matrix"), p + "o": ((w, nh * vd), "matrix")})
        else:
            nh, g, d, vd = (int(m["left"][k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            lp, rp = p + "left.", p + "right."
            out.update({lp + "q": ((nh * d, w), "matrix"), lp + "k": ((g * d, w), "matrix"), lp + "v": ((g * vd, w), "matrix"),
                        lp + "g": ((nh, w), "matrix"), lp + "o": ((w, nh * vd), "matrix")})
            rh, rd, rv = (int(m["right"][k]) for k in ("heads", "dim", "vdim"))
            out.update({rp + "q": ((rh * rd, w), "matrix"), rp + "k": ((rh * rd, w), "matrix"), rp + "v": ((rh * rv, w), "matrix"),
                        rp + "g": ((rh * rv, w), "matrix"), rp + "o": ((w, rh * rv), "matrix"), rp + "norm": ((rh * rv,), "norm"),
                        rp + "i": ((rh, w), "matrix"), rp + "i.b": ((rh,), "bonus"), rp + "f": ((rh, w), "matrix"),
                        rp + "f.b": ((rh,), "forget_base")})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        p = f"l{i}.mlp."
        out.update({f"l{i}.norm2": ((), "norm"), f"l{i}.ls2": ((w,), "norm")})
        if mlp["kind"] == "dense":
            out.update({p + "up": ((int(mlp["ff"]), w), "matrix"), p + "down": ((w, int(mlp["ff"])), "matrix")})
            continue
        ff, experts = int(mlp["expert"]["ff"]), int(mlp["router"]["experts"])
        for e in range(experts):
            out.update({f"{p}e{e}.up": ((ff, w), "matrix"), f"{p}e{e}.down": ((w, ff), "matrix")})
        out.update({p + "router": ((experts, w), "matrix"), p + "correction": ((experts,), "small")})
    out["final.norm"] = ((), "norm")
    out["head"] = ((cfg.vocab, w), "matrix")
    return out


register_architecture(["Mevuvik", "mevuvik"], MevuvikConfig, build_plan, checkpoint_layout)
