"""Fezozen on the GPU against the plain implementation: each mechanism's kernels alone, then whole
models through the trace runner, the step function and the generation entry point, with prompts cut
in every way, batches of unequal requests, reused slots and pages, keys that matter far back, at page
borders and at the two sides of a window's edge, long decoding and the first tokens of a sequence."""
import json
import os

import numpy as np
import pytest
import torch

import plain_fezozen as plain
from replay_util import Trace, run_trace
from tiny_configs import (FEZOZEN_A, FEZOZEN_B, FEZOZEN_C, _fezozen_attention, _fezozen_latent, _fezozen_moe, _fezozen_rot,
                          _fezozen_unit)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL_F32 = 3e-5
# bfloat16 engine against the float64 plain implementation, as a fraction of the largest logit
TOL_BF16 = 3e-2
PAGE = 64


def _dt(name):
    return torch.float32 if name == "float32" else torch.bfloat16


def _rand(rng, shape, dtype=torch.float32, scale=1.0, shift=0.0):
    """Random values that ``dtype`` holds exactly, as (device tensor, float64 numpy)."""
    t = torch.from_numpy(rng.standard_normal(shape) * scale + shift).to(dtype)
    return t.to(DEV), t.double().numpy()


def _i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def _packed(lens, slots, starts=None):
    """Index tensors of a packed step: (cu_seqlens, tok_seq, seq_slot, tok_pos)."""
    starts = starts or [0] * len(lens)
    cu = np.concatenate([[0], np.cumsum(lens)])
    seq = np.repeat(np.arange(len(lens)), lens)
    pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, lens)])
    return _i32(cu), _i32(seq), _i32(slots), _i32(pos)


def _steps(lens, sizes):
    """Walks sequences of ``lens`` tokens side by side in portions of ``sizes`` (the last size goes on):
    yields, step by step, [(sequence, lo, hi)] of the sequences that still have tokens."""
    at, k = [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        size = sizes[min(k, len(sizes) - 1)]
        live = [(i, at[i], min(n, at[i] + size)) for i, n in enumerate(lens) if at[i] < n]
        yield live
        for i, _, hi in live:
            at[i] = hi
        k += 1


def _inv_freq(rot):
    f, stretch = plain.frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    return (torch.from_numpy(f).float().to(DEV) if rot["dims"] else None), stretch


SCALED = {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}


# ------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,groups,dim,vdim,rot,scaling,unit", [
    (6, 2, 20, 12, 12, None, True), (4, 4, 24, 28, 16, SCALED, False), (3, 1, 64, 40, 64, None, True), (8, 2, 64, 64, 32, SCALED, False),
    (2, 1, 130, 130, 130, SCALED, True), (1, 1, 512, 8, 2, None, True), (5, 5, 7, 9, 0, None, True), (16, 4, 128, 128, 64, SCALED, False),
    (4, 2, 88, 56, 40, None, False)])
def test_rotated_pairs_and_unit_heads_into_the_cache(dtype, heads, groups, dim, vdim, rot, scaling, unit):
    """The kernel between the projection and the attention: q out, keys and values into their pages;
    sequences that start at positions 0, 61 (a page border inside the step), 300 and 63, in slots out of order."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads + dim)
    lens, starts, slots = [7, 9, 1, 70], [0, 61, 300, 63], [1, 0, 3, 2]
    cu, seq, slot, pos = _packed(lens, slots, starts)
    t, eps, r = sum(lens), 1e-3, _fezozen_rot(700.0, rot)
    if scaling:
        r["scaling"] = scaling
    u, un = _rand(rng, (t, (heads + groups) * dim + groups * vdim + 3), _dt(dtype))
    inv, stretch = _inv_freq(r)
    table = torch.randperm(24, generator=torch.Generator().manual_seed(1)).to(torch.int32).to(DEV).reshape(4, 6)
    kc = torch.zeros((24, groups, PAGE, dim), dtype=_dt(dtype), device=DEV)
    vc = torch.zeros((24, groups, vdim, PAGE), dtype=_dt(dtype), device=DEV)
    q = torch.empty((t, heads * dim), dtype=_dt(dtype), device=DEV)
    c = (heads + groups) * dim + groups * vdim
    kernels.filter_rope_cache(u[:, :c], None, None, inv, rot, pos, seq, slot, cu, table, PAGE, q, kc, vc, heads, groups, dim, vdim,
                              norm_eps=eps if unit else 0.0, rot_magnitude=stretch, pairs=True, unit_after=unit)

    def turned(x, n):
        y = plain.rotate_pairs(x.reshape(t, n, dim), pos.cpu().numpy(), r)
        return plain.unit_rms(y, eps) if unit else y

    tol = 4e-5 if dtype == "float32" else 1e-2
    want_q, want_k = turned(un[:, :heads * dim], heads), turned(un[:, heads * dim:(heads + groups) * dim], groups)
    want_v = un[:, (heads + groups) * dim:c].reshape(t, groups, vdim)
    assert np.abs(q.double().cpu().numpy().reshape(t, heads, dim) - want_q).max() < tol * np.abs(want_q).max()
    k, v = kc.double().cpu().numpy(), vc.double().cpu().numpy()
    pages = table.cpu().numpy()
    for i in range(t):
        page, off = pages[slots[int(seq[i])], int(pos[i]) // PAGE], int(pos[i]) % PAGE
        assert np.abs(k[page, :, off] - want_k[i]).max() < tol * np.abs(want_k).max()
        assert np.array_equal(v[page, :, :, off], want_v[i])
    touched = {(int(pages[slots[int(seq[i])], int(pos[i]) // PAGE]), int(pos[i]) % PAGE) for i in range(t)}
    rest = np.ones((24, PAGE), bool)
    for page, off in touched:
        rest[page, off] = False
    assert not k.transpose(0, 2, 1, 3)[rest].any() and not v.transpose(0, 3, 1, 2)[rest].any()      # nothing else was written


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rd,rank", [(3, 24, 12, 44), (4, 32, 16, 80), (1, 0, 10, 20), (2, 16, 6, 96)])
def test_latent_rows_with_stretched_rotation(dtype, heads, dim, rd, rank):
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads + rank)
    lens, starts, slots = [7, 9, 1], [0, 61, 300], [1, 0, 2]
    cu, seq, slot, pos = _packed(lens, slots, starts)
    t, r = sum(lens), {**_fezozen_rot(700.0, rd), "scaling": SCALED}
    q, qn = _rand(rng, (t, heads * (dim + rd)))
    kv, kvn = _rand(rng, (t, rank + rd + 5))
    w, wn = _rand(rng, (rank,), shift=1.0, scale=0.2)
    inv, stretch = _inv_freq(r)
    table = torch.arange(3 * 6, dtype=torch.int32, device=DEV).reshape(3, 6)
    cache = torch.zeros((18, PAGE, rank + rd), dtype=_dt(dtype), device=DEV)
    q_nope = torch.empty((t, heads * dim), dtype=_dt(dtype), device=DEV)
    qa = torch.zeros((t, heads * (rank + rd)), dtype=_dt(dtype), device=DEV)
    kernels.latent_prepare(q, kv[:, :rank + rd], None, w, 1e-5, inv, rd, 0.3, q_nope, qa, None, cache, table, PAGE, pos, seq, slot,
                           heads, dim, rd, rank, rot_magnitude=stretch)
    tol = 4e-5 if dtype == "float32" else 1e-2
    p = pos.cpu().numpy()
    got = qa.double().cpu().numpy().reshape(t, heads, rank + rd)[..., rank:]
    want = plain.rotate_pairs(qn.reshape(t, heads, dim + rd)[..., dim:] * 0.3, p, r)
    assert np.abs(got - want).max() < tol * np.abs(want).max()
    rows = np.concatenate([plain.rms_norm(kvn[:, :rank], wn, 1e-5), plain.rotate_pairs(kvn[:, None, rank:rank + rd], p, r)[:, 0]], axis=1)
    held = cache.double().cpu().numpy()
    for i in range(t):
        page = int(table[slots[int(seq[i])], int(p[i]) // PAGE])
        assert np.abs(held[page, int(p[i]) % PAGE] - rows[i]).max() < tol * np.abs(rows).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("t,heads,n,k,pad", [(1, 3, 20, 44, 1), (8, 16, 64, 128, 0), (70, 5, 33, 24, 3), (200, 4, 128, 256, 0), (9, 2, 130, 72, 2)])
def test_products_of_heads_with_a_gate_per_number(dtype, t, heads, n, k, pad):
    from gemmars_b200 import kernels
    rng = np.random.default_rng(t + n)
    x, xn = _rand(rng, (t, heads, k), _dt(dtype))
    w, wn = _rand(rng, (heads, n, k), _dt(dtype), scale=k ** -0.5)
    z, zn = _rand(rng, (t, heads * n + pad), scale=3.0)
    s, sn = _rand(rng, (t, heads), shift=1.0)
    full = np.einsum("thk,hnk->thn", xn, wn)
    gate = plain.sigmoid(zn[:, pad:].reshape(t, heads, n))
    for scale in (None, s):
        y = torch.empty((t, heads, n), dtype=_dt(dtype), device=DEV)
        kernels.heads_gemm(x, w, y, heads, scale=scale, gate=z[:, pad:])
        want = full * gate * (1.0 if scale is None else sn[:, :, None])
        assert np.abs(y.double().cpu().numpy() - want).max() < (3e-5 if dtype == "float32" else 1e-2) * np.abs(want).max()


def _part(category, kind, params, tensors, dtype):
    from gemmars_b200.parts.base import build_part
    from gemmars_b200.parts.plan import PartSpec
    part = build_part(category, PartSpec(kind, params, {k: k for k in tensors}), dtype)
    wants = part.wants()
    assert set(wants) == set(tensors)
    part.load({k: (v.to(_dt(dtype)) if wants[k].role == "matrix" else v.float()) for k, v in tensors.items()})
    return part


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("t,width,experts,top,ff", [(1, 64, 4, 2, 32), (9, 52, 3, 3, 20), (15, 72, 6, 1, 40), (40, 64, 5, 2, 48),
                                                    (255, 128, 16, 4, 64), (300, 128, 9, 3, 72), (700, 64, 4, 4, 32), (513, 192, 11, 1, 130)])
def test_raw_sigmoid_routing_of_weighted_inputs(dtype, t, width, experts, top, ff):
    """Token-major (fewer than 16 tokens, and float32), grouped (16 to 255) and on the tcgen05 product (256
    and more), added into a stream and stored into rows of its own.  The gate's argument is large enough
    that a weight on the output instead of the input shows."""
    rng = np.random.default_rng(t + experts)
    w, wn = {}, {}

    def add(name, shape, scale):
        w[name], wn[name] = _rand(rng, shape, torch.bfloat16, scale=scale)

    add("router", (experts, width), 0.25)
    for e in range(experts):
        add(f"e{e}.gate", (ff, width), 0.3)
        add(f"e{e}.up", (ff, width), 0.25)
        add(f"e{e}.down", (width, ff), 0.1)
    params = {"hidden_size": width, "experts": experts, "top": top, "ff": ff, "limit": None, "alpha": 1.0, "shift": 0.0,
              "router_bias": False, "routing": "sigmoid_raw", "weigh": "input", "shared": None}
    h, hn = _rand(rng, (t, width), _dt(dtype))
    base, basen = _rand(rng, (t, width), torch.float32)
    mlp = {"router": {"experts": experts, "top": top}}
    out = plain.routed_ffn(hn, wn, mlp)
    on_output = np.zeros_like(out)
    z = hn @ wn["router"].T
    for i in range(t):
        for e, s in zip(*plain.choose(z[i], top)):
            on_output[i] += s * plain.expert(hn[i], wn, e)
    assert np.abs(out - on_output).max() > 0.05 * np.abs(out).max()
    # a token whose last chosen and first unchosen scores are closer than rounding may go either way
    c = np.sort(plain.sigmoid(z), axis=1)[:, ::-1]
    sure = np.ones(t, bool) if top == experts else (c[:, top - 1] - c[:, top]) > 1e-5       # both precisions hold the inputs exactly
    assert sure.mean() > 0.9
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    for store in (False, True):
        part = _part("ffn", "moe", params, w, dtype)
        if store:
            part.set_output_store()
        res = base.clone()
        part.forward(type("Ctx", (), dict(host=None))(), h, res)
        want = out if store else basen + out
        assert np.abs(res.double().cpu().numpy() - want)[sure].max() <= tol * np.abs(want).max(), store
    from gemmars_b200 import kernels
    kernels.check_status()


def _attention_case(rng, total, heads, groups, dim, vdim, dt, spots):
    """q of one new token (or the last of several), keys and values; the keys at ``spots`` all score high for
    head 0's last query, each with a value of its own."""
    q, _ = _rand(rng, (total, heads, dim), dt)
    k, _ = _rand(rng, (total, groups, dim), dt, scale=0.3)
    v, _ = _rand(rng, (total, groups, vdim), dt)
    q[-1] = 0.0
    q[-1, :, 0] = 8.0
    for p in spots:
        k[p] = 0.0
        k[p, :, 0] = 8.0
    return q, k, v


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(3, 1, 20, 12), (8, 2, 64, 40), (4, 4, 128, 128), (6, 2, 32, 64), (16, 1, 64, 128)])
@pytest.mark.parametrize("window,cap", [(64, 0.0), (65, 20.0), (100, 0.0), (1, 0.0), (None, 30.0)])
def test_window_edges_alone(dtype, heads, groups, dim, vdim, window, cap):
    """The key just inside the window and the one just outside carry all the score: a window that is one
    off reads the other's value.  In a prompt (from position 0 and in portions) and as a single token."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads * 7 + (window or 0))
    total, dt = 230, _dt(dtype)
    first = total - window if window else 0
    q, k, v = _attention_case(rng, total, heads, groups, dim, vdim, dt, [p for p in (first, first - 1) if 0 <= p < total - 1])
    qn, kn, vn = (x.double().cpu().numpy() for x in (q, k, v))
    full = plain.masked_attention(qn, kn, vn, 0.25, cap, window)
    if window and window > 1:
        assert np.abs(full[-1, 0] - vn[first, 0]).max() < 0.05               # all of it is the edge's value
    table = _i32([[4, 2, 3, 1]])
    kc = torch.zeros((6, groups, PAGE, dim), dtype=dt, device=DEV)
    vc = torch.zeros((6, groups, vdim, PAGE), dtype=dt, device=DEV)
    for p in range(total):
        page = int(table[0, p // PAGE])
        kc[page, :, p % PAGE], vc[page, :, :, p % PAGE] = k[p], v[p]
    for new in (total, 70, 2, 1):
        cu, seq, slot, pos = _packed([new], [0], [total - new])
        ctx = type("Ctx", (), dict(cu_seqlens=cu, seq_start=_i32([total - new]), seq_slot=slot, n_seqs=1, tok_pos=pos, tok_seq=seq,
                                   max_new=new, max_total=total, host=None))()
        out = torch.empty((new, heads * vdim), dtype=dt, device=DEV)
        kernels.attention_capped(ctx, q[total - new:].reshape(new, -1), out, heads, kc, vc, table, PAGE, window, 0.25, cap)
        got = out.double().cpu().numpy().reshape(new, heads, vdim)
        assert np.abs(got - full[total - new:]).max() < (2e-5 if dtype == "float32" else 2e-2) * np.abs(full).max(), new
    kernels.check_status()


@pytest.mark.parametrize("dim,vdim", [(64, 64), (128, 128), (24, 32), (48, 80)])
@pytest.mark.parametrize("window,cap,sink,gate", [(None, 0.0, False, None), (100, 3.0, False, None), (None, 2.0, True, "number"),
                                                  (65, 0.0, True, "head")])
def test_batches_of_prompts_and_of_single_tokens(dim, vdim, window, cap, sink, gate):
    """bfloat16 attention over scattered pages: prompts and portions of unequal lengths in one step (the
    tcgen05 kernel), and steps of 1, 4 and 20 single tokens (a head's keys dealt to clusters of 8, 8 and 2
    CTAs) and of 60 (to none), with everything that may happen to the scores and to the result."""
    from gemmars_b200 import kernels
    dt, heads, groups = torch.bfloat16, 6, 2
    for lens, starts in (([150, 33, 1, 300], [0, 70, 300, 1]), ([1], [333]), ([1] * 4, [0, 64, 1000, 130]),
                         ([1] * 20, [37 * i for i in range(20)]), ([1] * 60, [7 * i for i in range(60)])):
        rng = np.random.default_rng(len(lens))
        n, t = len(lens), sum(lens)
        cu, seq, slot, pos = _packed(lens, list(range(n))[::-1], starts)
        wide = max(-(-(a + b) // PAGE) for a, b in zip(lens, starts))
        table = torch.randperm(n * wide, generator=torch.Generator().manual_seed(n)).to(torch.int32).reshape(n, wide)
        kc, kn = _rand(rng, (n * wide, groups, PAGE, dim), dt)
        vc, vn = _rand(rng, (n * wide, groups, vdim, PAGE), dt)
        q, qn = _rand(rng, (t, heads * dim), dt)
        s, sn = _rand(rng, (heads,), scale=3.0)
        g, gn = _rand(rng, (t, heads if gate == "head" else heads * vdim), dt)
        ctx = type("Ctx", (), dict(cu_seqlens=cu, seq_start=_i32(starts), seq_slot=slot, n_seqs=n, tok_pos=pos, tok_seq=seq,
                                   max_new=max(lens)))()
        out = torch.zeros((t, heads * vdim), dtype=dt, device=DEV)
        kernels.attention_capped(ctx, q, out, heads, kc, vc, table.to(DEV), PAGE, window, 0.8 * dim ** -0.5, cap, g if gate else None,
                                 1.3, 0, s if sink else None, gate == "head")
        kernels.check_status()
        got = out.double().cpu().numpy().reshape(t, heads, vdim)
        at = 0
        for i in range(n):
            total = starts[i] + lens[i]
            pages = table[n - 1 - i].numpy()[:-(-total // PAGE)]
            k = kn[pages].transpose(0, 2, 1, 3).reshape(-1, groups, dim)[:total]
            v = vn[pages].transpose(0, 3, 1, 2).reshape(-1, groups, vdim)[:total]
            seen = plain.visible(total, window)[starts[i]:]
            x = qn[at:at + lens[i]].reshape(lens[i], heads, dim)
            for h in range(heads):
                sc = np.where(seen, plain.capped((x[:, h] @ k[:, h // 3].T) * 0.8 * dim ** -0.5, cap), -np.inf)
                e = np.exp(sc)
                want = 1.3 * (e @ v[:, h // 3]) / (e.sum(axis=1, keepdims=True) + (np.exp(sn[h]) if sink else 0.0))
                if gate == "head":
                    want *= plain.sigmoid(gn[at:at + lens[i], h:h + 1])
                elif gate:
                    want *= plain.sigmoid(gn[at:at + lens[i], h * vdim:(h + 1) * vdim])
                assert np.abs(got[at:at + lens[i], h] - want).max() < 1.5e-2 * max(1.0, np.abs(want).max()), (lens[i], h)
            at += lens[i]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("raw,layer", [(FEZOZEN_A, 1), (FEZOZEN_B, 0), (FEZOZEN_B, 3)], ids=["A1", "B0", "B3"])
def test_latent_mixer_alone(dtype, raw, layer, monkeypatch):
    """The latent mixer from its input to its output: whole prompts of 300 tokens (expanded per head where
    the sizes allow), the same with the expansion off, in portions, and token by token, with the window
    moving on; the gates' logits are spread so that a lost gate shows."""
    from gemmars_b200 import kernels
    from gemmars_b200.cache.pool import KVGroup
    from gemmars_b200.models.fezozen import FezozenConfig, _latent_spec
    from gemmars_b200.parts.base import build_part
    cfg, m = FezozenConfig.from_dict(raw), raw["layers"][layer]["mixer"]
    spec = _latent_spec(cfg, m, "")
    part = build_part("mixer", spec, dtype)
    rng = np.random.default_rng(layer)
    w, wn = {}, {}
    for short, want in part.wants().items():
        big = {"q": 0.25, "dkv": 0.25, "g": 0.3, "uk": 0.4}.get(short, 0.2)
        w[short], arr = _rand(rng, want.shape, torch.bfloat16, scale=big, shift=1.0 if short == "dkv_norm" else 0.0)
        wn[spec.tensors[short]] = arr
    part.load({k: (x.to(_dt(dtype)) if part.wants()[k].role == "matrix" else x.float()) for k, x in w.items()})
    n, width = 300, cfg.width
    h, hn = _rand(rng, (n, width), _dt(dtype))
    want = plain.latent_attention_mixer(hn, wn, m, cfg.norm_eps)
    lost = plain.latent_attention_mixer(hn, {**wn, "g": 0 * wn["g"]}, m, cfg.norm_eps)
    longer = plain.latent_attention_mixer(hn, wn, {**m, "mask": {"size": m["mask"]["size"] + 1}}, cfg.norm_eps)
    assert np.abs(lost - want).max() > 0.2 * np.abs(want).max() and np.abs(longer - want).max() > 0.05 * np.abs(want).max()

    def run(sizes):
        group = KVGroup(part.cache_needs()[0], 1, 2, 32, 16, n, _dt(dtype), DEV)
        out = torch.zeros((n, width), dtype=torch.float32, device=DEV)
        for live in _steps([n], sizes):
            (_, lo, hi), = live
            group.reserve(1, hi)
            group.sync()
            cu, seq, slot, pos = _packed([hi - lo], [1], [lo])
            ctx = type("Ctx", (), dict(cu_seqlens=cu, seq_start=_i32([lo]), seq_slot=slot, n_seqs=1, tok_pos=pos, tok_seq=seq,
                                       max_new=hi - lo, max_total=hi, host={"seq_start": [lo], "seq_len": [hi - lo], "seq_slot": [1]}))()
            part.forward(ctx, h[lo:hi], out[lo:hi], [(group, *group.layer(0))])
        return out.double().cpu().numpy()

    tol = (3e-5 if dtype == "float32" else 2.5e-2) * np.abs(want).max()
    assert kernels.latent_expand_usable(torch.bfloat16, m["kv_rank"], m["dim"], m["rot_dim"], m["vdim"]) == (layer == 0)
    for sizes in ([n], [2, 64, 130, 100], [1]):
        assert np.abs(run(sizes) - want).max() < tol, sizes
    monkeypatch.setattr(kernels, "LATENT_EXPAND_MIN_TOKENS", n + 1)
    assert np.abs(run([n]) - want).max() < tol


def test_stored_rows_are_the_products_alone():
    """A product that stores: every way a product takes, into rows that held something else."""
    from gemmars_b200.parts.linear import Linear
    rng = np.random.default_rng(5)
    for m, n, k in ((1, 512, 2048), (7, 96, 128), (40, 72, 512), (65, 200, 128), (300, 520, 200), (5, 50, 52)):
        for dtype in ("float32", "bfloat16"):
            x, xn = _rand(rng, (m, k), _dt(dtype))
            w, wn = _rand(rng, (n, k), _dt(dtype), scale=k ** -0.5)
            b, bn = _rand(rng, (n,))
            lin = Linear(w, b)
            lin.stores = True
            rows, _ = _rand(rng, (m, n), scale=5.0)
            assert lin.add_into(x, rows) is None
            want = xn @ wn.T + bn
            assert np.abs(rows.double().cpu().numpy() - want).max() < 3e-5 * np.abs(want).max(), (m, n, k, dtype)
            lin.out_scale = b
            with pytest.raises(ValueError):
                lin.add_into(x, rows)


# ------------------------------------------------------------------ whole models

def _sharp_folder(tmp_path_factory, raw, seed, factor):
    """Random weights whose attention queries and keys are scaled by ``factor``: scores grow with its
    square, the softmax picks single keys instead of averaging, and a wrong key, page, slot or rotation
    shows in the logits.  Biases, routers, gates and experts are loud as well."""
    from gemmars_b200.weights import random_weights, write_safetensors
    tensors = random_weights(raw, seed=seed)
    for name in tensors:
        by = 1.0
        if name.endswith((".mix.q", ".mix.k", ".mix.uk", ".mix.dkv")):
            by = factor
        elif name.endswith(".b"):
            by = 15.0
        elif name.endswith(".mix.g"):
            by = 12.0
        elif name.endswith((".mix.v", ".mix.uv", ".gate", ".up")):
            by = 8.0
        elif name.endswith(".router"):
            by = 8.0
        elif name == "head":
            by = 12.0
        if by != 1.0:
            tensors[name] = (tensors[name].float() * by).bfloat16()
    d = str(tmp_path_factory.mktemp("fezozen"))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(raw, f)
    write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d


def _within(errors, tol, what, share=0.0):
    """Every position within ``tol``, but for a ``share`` of them."""
    errors = np.asarray(errors)
    over = int((errors > tol).sum())
    assert over <= int(share * errors.size), f"{what}: {over} of {errors.size} positions are over {tol:.2e} (worst {errors.max():.2e})"


REQUESTS = {"A": (FEZOZEN_A, [15, 21, 9, 70, 44, 131]), "B": (FEZOZEN_B, [17, 33, 3, 80, 150, 300])}
GROUPS = [[0, 1, 2], [3, 4, 5]]


def _every_expert(raw):
    """The configuration with every expert chosen.  Rounding a router's input now and then sends a token whose
    candidates have nearly equal scores to another expert; a sublayer's output is normed, so that token's
    stream is then another one altogether, and with sharp attention so are its readers'.  What the
    choice is, is tested alone and in float32; the bfloat16 models below leave nothing to choose, so
    that every position can be held to a tolerance."""
    layers = []
    for layer in raw["layers"]:
        mlp = layer["mlp"]
        if mlp is not None:
            mlp = {**mlp, "router": {**mlp["router"], "top": mlp["router"]["experts"]}}
        layers.append({**layer, "mlp": mlp})
    return {**raw, "layers": layers}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (raw, lengths) in REQUESTS.items():
        for dtype in ("float32", "bfloat16"):
            mine = raw if dtype == "float32" else _every_expert(raw)
            folder = _sharp_folder(tmp_path_factory, mine, seed=32, factor={"A": (9.0, 5.0), "B": (5.0, 3.5)}[name][dtype == "bfloat16"])
            cfg, w = plain.load_folder(folder)
            rng = np.random.default_rng(lengths[0])
            reqs = [rng.integers(0, raw["vocab"], n).tolist() for n in lengths]
            out[name, dtype] = (folder, cfg, w, reqs, [plain.forward(cfg, w, r) for r in reqs])
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_test_models_show_a_fault(dtype, models):
    """The scaled weights do what they are for: in the plain model, queries turned one position too far, a
    lost first key, windows one longer or shorter, a cap left out, rotations without their stretch, unit
    heads or gates left out, or a weight on the expert's output move the logits by far more than rounding."""
    folder, cfg, w, reqs, ref = models["A", dtype]
    toks = reqs[5]
    scale = np.abs(ref[5]).max()

    def planted(name, fault):
        saved = getattr(plain, name)
        try:
            setattr(plain, name, fault(saved))
            return plain.forward(cfg, w, toks)
        finally:
            setattr(plain, name, saved)

    def on_output(inner):
        return lambda h, P, mlp: np.stack([sum(s * plain.expert(h[t], P, e) for e, s in zip(*plain.choose(h[t] @ P["router"].T, mlp["router"]["top"])))
                                           for t in range(h.shape[0])])

    runs = {"rotation": planted("rotate_pairs", lambda f: lambda x, pos, rot: f(x, np.asarray(pos) + (x.shape[1] > 2), rot)),
            "first key": planted("masked_attention", lambda f: lambda q, k, v, *a: f(q, np.concatenate([0 * k[:1], k[1:]]), v, *a)),
            "window +1": planted("window_of", lambda f: lambda m: f(m) and f(m) + 1),
            "window -1": planted("window_of", lambda f: lambda m: f(m) and f(m) - 1),
            "cap": planted("capped", lambda f: lambda z, c: z),
            "stretch": planted("frequencies", lambda f: lambda *a: (f(*a)[0], 1.0)),
            "unit": planted("MIXERS", lambda f: {**f, "attention_2": lambda h, P, m, eps: plain.biased_attention_mixer(
                h, {**P, "q.b": 0.0, "k.b": 0.0, "v.b": 0.0}, m, eps)}),
            "gate": planted("output_gate", lambda f: lambda h, g: np.full((h.shape[0], g.shape[0]), 0.5)),
            "weights": planted("routed_ffn", on_output)}
    for what, other in runs.items():
        moved = np.abs(other - ref[5]).max(axis=1)
        assert moved.max() > 2 * TOL_BF16 * scale and (moved[40:] > 100 * TOL_F32 * scale).mean() > 0.3, (what, moved.max() / scale)


@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_all_cuttings_match_the_plain_implementation(name, dtype, models, tmp_path):
    """Through bin/trace_run: each request whole, with its last 40 tokens one by one, and in two batches of
    unequal requests that follow one another in a cache sized to the peak, so that the second batch
    lives in the slots and pages the first gave back."""
    folder, cfg, w, reqs, ref = models[name, dtype]
    tr = Trace()
    tr.whole("w", reqs)
    tr.tail("t", reqs, n_tail=40)
    prompt_lens = [max(1, len(r) - 8 - 3 * i) for i, r in enumerate(reqs)]
    prompt_lens[2] = len(reqs[2])
    prompt_lens[1] = 1
    tr.batches("b", reqs, GROUPS, prompt_lens)
    got = run_trace(tr, folder, dtype, str(tmp_path / "out"))
    scale = max(float(np.abs(r).max()) for r in ref)
    tol = (TOL_F32 if dtype == "float32" else TOL_BF16) * scale
    for tag in "wtb":
        _within([np.abs(got[(f"{tag}{i}", p)] - r[p]).max() for i, r in enumerate(ref) for p in range(len(r))], tol, f"cutting {tag!r}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_after_every_run_of_a_layer(dtype, models):
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, _ = models["A", dtype]
    toks = reqs[3]
    _, want = plain.forward(cfg, w, toks, return_layers=True)
    model = build_model(folder, dtype=dtype)
    assert len(model.blocks) == 4 and len(model.plan.schedule) == 6 == len(want)
    seen, given = [], []
    for block in model.blocks:
        def run(ctx, x, caches, _inner=block.forward, **kw):
            given.append(kw.get("h_in") is not None)
            left = _inner(ctx, x, caches, **kw)
            assert x.dtype == torch.float32                      # the residual stream is 32-bit in both modes
            seen.append(x.double().cpu().numpy())
            return left
        block.forward = run
    runner = Runner(model, max_tokens=256, max_batch=1, use_graphs=False)
    runner.step([StepItem(runner.open(), toks, [])])
    assert len(seen) == len(want) and given == [False] + [True] * 5      # each layer's last norm leaves the next one's first
    for i, (a, b) in enumerate(zip(seen, want)):
        tol = (1e-5 if dtype == "float32" else 2e-2) * np.abs(b).max()
        _within(np.abs(a - b).max(axis=1), tol, f"run {i}")


@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_long_decoding_and_reused_slots(name, dtype, models):
    """One runner, a cache of eight pages.  A prompt in portions of 2, 3, 64, 1, 65 and the rest;
    another from its first token one by one for 300 steps, across four page borders and every window,
    beside a neighbour that comes and goes; then the same again in the slots and pages given back: in
    float32 to the last bit."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, ref = models[name, dtype]
    model = build_model(folder, dtype=dtype)
    runner = Runner(model, max_tokens=8 * PAGE, max_batch=3)
    rng = np.random.default_rng(8)
    long_toks = rng.integers(0, cfg["vocab"], 300).tolist()
    long_ref = plain.forward(cfg, w, long_toks)
    scale = float(np.abs(long_ref).max())
    tol = (TOL_F32 if dtype == "float32" else TOL_BF16) * scale
    first_round = None
    for round_ in range(2):
        got = {}
        a = runner.open()
        at = 0
        for n in (2, 3, 64, 1, 65, 15):
            part = reqs[4][at:at + n]
            if not part:
                break
            got.update({("a", at + i): r for i, r in enumerate(runner.step([StepItem(a, part, range(len(part)))]).cpu().numpy())})
            at += len(part)
        assert at == len(reqs[4])
        runner.close(a)
        b = runner.open()
        c = None
        for p, tok in enumerate(long_toks):
            items = [StepItem(b, [tok], [0])]
            if p == 20:
                c = runner.open()
                items.append(StepItem(c, reqs[0], range(len(reqs[0]))))     # a prompt beside a decoded token
            elif c is not None and p < 20 + 30:
                items.append(StepItem(c, [reqs[1][(p - 21) % len(reqs[1])]], [0]))
            out = runner.step(items).cpu().numpy()
            got[("b", p)] = out[0]
            if p == 20:
                got.update({("c", i): r for i, r in enumerate(out[1:])})
            if p == 49:
                runner.close(c)
                c = None
        runner.close(b)
        assert runner.cache.pages_held() == 0
        _within([np.abs(got[("a", p)] - ref[4][p]).max() for p in range(len(reqs[4]))], tol, "portions")
        _within([np.abs(got[("b", p)] - long_ref[p]).max() for p in range(len(long_toks))], tol, "decoded")
        _within([np.abs(got[("c", p)] - ref[0][p]).max() for p in range(len(reqs[0]))], tol, "neighbour")
        if first_round is None:
            first_round = got
        elif dtype == "float32":
            assert all(np.array_equal(got[k], first_round[k]) for k in got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_the_tensor_cores_do_not_take(dtype, tmp_path_factory):
    """A width of 52 and heads of 20, 12, 9, 6 and 5, a window of one key: every product and the attention
    run on the plain kernels.  Prompts in portions of two tokens, then token by token, against the whole."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    raw = FEZOZEN_C if dtype == "float32" else _every_expert(FEZOZEN_C)
    folder = _sharp_folder(tmp_path_factory, raw, seed=5, factor=10.0 if dtype == "float32" else 5.0)
    cfg, w = plain.load_folder(folder)
    rng = np.random.default_rng(13)
    reqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (61, 2, 30)]
    ref = [plain.forward(cfg, w, r) for r in reqs]
    scale = max(float(np.abs(r).max()) for r in ref)
    runner = Runner(build_model(folder, dtype=dtype), max_tokens=4 * PAGE, max_batch=3)
    slots = [runner.open() for _ in reqs]
    errs = []
    for live in _steps([len(r) for r in reqs], [2, 2, 2, 2, 1]):
        out = runner.step([StepItem(slots[i], reqs[i][lo:hi], range(hi - lo)) for i, lo, hi in live]).cpu().numpy()
        at = 0
        for i, lo, hi in live:
            errs += list(np.abs(out[at:at + hi - lo] - ref[i][lo:hi]).max(axis=1))
            at += hi - lo
    assert len(errs) == sum(len(r) for r in reqs)
    _within(errs, (TOL_F32 if dtype == "float32" else TOL_BF16) * scale, "portions of two")
    for s in slots:
        runner.close(s)
    assert runner.cache.pages_held() == 0


def test_long_prompts_on_the_tensor_cores(models):
    """Prompts of more than 256 tokens: keys and values expanded per head under a window, experts on the
    tcgen05 product; one alone, two in one step, one in two portions (the second reads the latent rows
    of the first)."""
    from gemmars_b200 import kernels
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, _ = models["B", "bfloat16"]
    rng = np.random.default_rng(7)
    runner = Runner(build_model(folder, dtype="bfloat16"), max_tokens=20 * PAGE, max_batch=2)
    toks = [rng.integers(0, cfg["vocab"], n).tolist() for n in (301, 457)]
    want = [plain.forward(cfg, w, t) for t in toks]
    scale = max(np.abs(x).max() for x in want)
    slots = [runner.open() for _ in toks]
    out = runner.step([StepItem(s, t, range(len(t))) for s, t in zip(slots, toks)]).cpu().numpy()
    errs = list(np.abs(out[:301] - want[0]).max(axis=1)) + list(np.abs(out[301:] - want[1]).max(axis=1))
    for s in slots:
        runner.close(s)
    s = runner.open()
    out = np.concatenate([runner.step([StepItem(s, toks[1][a:b], range(b - a))]).cpu().numpy() for a, b in ((0, 130), (130, 457))])
    errs += list(np.abs(out - want[1]).max(axis=1))
    kernels.check_status()
    _within(errs, TOL_BF16 * scale, "long prompts")


def test_routed_models_in_bfloat16(tmp_path_factory):
    """Tokens that have experts to choose, with attention gentle enough that a token that went elsewhere stays
    nearly alone: whole prompts, the last tokens one by one, and both models' kinds of kernels."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    for raw, factor in ((FEZOZEN_A, 2.0), (FEZOZEN_B, 1.5)):
        folder = _sharp_folder(tmp_path_factory, raw, seed=8, factor=factor)
        cfg, w = plain.load_folder(folder)
        runner = Runner(build_model(folder, dtype="bfloat16"), max_tokens=8 * PAGE, max_batch=1)
        toks = np.random.default_rng(3).integers(0, raw["vocab"], 300).tolist()
        want = plain.forward(cfg, w, toks)
        s = runner.open()
        out = [runner.step([StepItem(s, toks[:270], range(270))]).cpu().numpy()]
        out += [runner.step([StepItem(s, [t], [0])]).cpu().numpy() for t in toks[270:]]
        errors = np.abs(np.concatenate(out) - want).max(axis=1)
        _within(errors, TOL_BF16 * np.abs(want).max(), f"routed, width {raw['width']}", share=0.15)
        assert np.median(errors) < 0.5 * TOL_BF16 * np.abs(want).max()


def _random_configuration(rng):
    """Layers of all kinds in any order with sizes drawn at random, some of which run another layer's tensors."""
    def scaling():
        return (float(rng.uniform(1.5, 10)), int(rng.choice([32, 100, 2048])), float(rng.choice([8.0, 32.0])), float(rng.choice([0.5, 1.0]))) \
            if rng.random() < 0.6 else None

    def mlp():
        if rng.random() < 0.15:
            return None
        experts = int(rng.integers(1, 13))
        return _fezozen_moe(experts, int(rng.integers(1, min(experts, 6) + 1)), int(rng.choice([24, 32, 40, 66, 96])))

    def mixer(kind):
        if kind == "latent_attention":
            dim, rd = int(rng.choice([4, 16, 24, 32, 64])), int(rng.choice([2, 8, 16, 20, 32]))
            return _fezozen_latent(int(rng.integers(1, 7)), dim, rd, int(rng.choice([8, 16, 20, 32, 48])), int(rng.choice([12, 32, 48, 80, 160])),
                                   float((dim + rd) ** -0.5 * rng.uniform(0.7, 1.5)), int(rng.choice([1, 5, 63, 64, 90, 400])),
                                   float(rng.choice([1e4, 3e5, 100.0])), scaling())
        g, dim = int(rng.choice([1, 2, 3])), int(rng.choice([12, 16, 32, 64, 80, 96]))
        heads, vdim = g * int(rng.choice([1, 2, 3, 5])), int(rng.choice([16, 40, 64, dim]))
        rot = _fezozen_rot(float(rng.choice([1e4, 1e6, 50.0])), 2 * int(rng.integers(1, dim // 2 + 1)), scaling())
        if kind == "attention":
            return _fezozen_attention(heads, g, dim, vdim, float(dim ** -0.5 * rng.uniform(0.7, 1.5)), float(rng.choice([5.0, 30.0])), rot)
        rot.pop("scaling", None)
        return _fezozen_unit(heads, g, dim, vdim, float(dim ** -0.5 * rng.uniform(1.0, 3.0)), int(rng.choice([1, 5, 63, 64, 65, 128, 400])), rot)

    layers = []
    for i in range(int(rng.integers(1, 7))):
        if layers and rng.random() < 0.3:
            j = int(rng.integers(0, len(layers)))
            layers.append({**layers[j], "weights_of": j})
            continue
        kind = str(rng.choice(["attention", "attention_2", "latent_attention"]))
        layers.append({"type": kind, "mixer": mixer(kind), "mlp": mlp()})
    return {"architecture": "Fezozen", "vocab": int(rng.choice([97, 300, 1000])), "width": int(rng.choice([52, 64, 96, 136, 200])),
            "embedding": {"scale": float(rng.choice([1.0, 0.3, 12.0]))}, "norm": {"eps": float(rng.choice([1e-5, 1e-6]))}, "layers": layers}


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_random_configurations(seed, tmp_path_factory):
    """A configuration drawn at random, in float32: three unequal prompts in one batch, then token by
    token together until the shortest ends and on, against the plain implementation's whole prompts."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    rng = np.random.default_rng(1000 + seed)
    raw = _random_configuration(rng)
    folder = _sharp_folder(tmp_path_factory, raw, seed=seed, factor=2.0)
    cfg, w = plain.load_folder(folder)
    lens = [int(n) for n in rng.choice([2, 17, 70, 131, 200], 3)]
    reqs = [rng.integers(0, raw["vocab"], n).tolist() for n in lens]
    ref = [plain.forward(cfg, w, r) for r in reqs]
    scale = max(float(np.abs(r).max()) for r in ref)
    runner = Runner(build_model(folder, dtype="float32"), max_tokens=12 * PAGE, max_batch=3)
    slots = [runner.open() for _ in reqs]
    heads = [max(1, n - 9) for n in lens]
    errs = []
    out = runner.step([StepItem(s, r[:h], range(h)) for s, r, h in zip(slots, reqs, heads)]).cpu().numpy()
    at = 0
    for r, h in zip(ref, heads):
        errs += list(np.abs(out[at:at + h] - r[:h]).max(axis=1))
        at += h
    for k in range(9):
        live = [i for i in range(3) if heads[i] + k < lens[i]]
        if not live:
            break
        out = runner.step([StepItem(slots[i], [reqs[i][heads[i] + k]], [0]) for i in live]).cpu().numpy()
        errs += [np.abs(out[n] - ref[i][heads[i] + k]).max() for n, i in enumerate(live)]
    assert len(errs) == sum(lens)
    assert max(errs) <= TOL_F32 * scale, f"{max(errs) / scale:.2e} of the largest logit, configuration {json.dumps(raw)}"
    for s in slots:
        runner.close(s)
    assert runner.cache.pages_held() == 0


def test_greedy_generation_through_the_engine(models):
    from gemmars_b200 import Engine
    folder, cfg, w, reqs, _ = models["A", "float32"]
    eng = Engine.load(folder, "dtype=float32;max_batch=3;max_tokens=2048")
    prompts = [reqs[0], reqs[2], [5], reqs[4][:33], reqs[3]]
    free_run, _ = plain.generate(cfg, w, prompts[0], 10)
    stop = [free_run[4]]
    res = eng.generate(prompts, max_tokens=10, stop_ids=stop)
    for p, r in zip(prompts, res):
        want, reason = plain.generate(cfg, w, p, 10, stop=stop)
        assert r.tokens == want and r.reason == reason
    assert eng.runner.cache.pages_held() == 0
    again = eng.generate(list(reversed(prompts)), max_tokens=10, stop_ids=stop)
    assert [r.tokens for r in reversed(again)] == [r.tokens for r in res]
    # bfloat16 decodes through captured steps: the tokens it picks are the plain model's best or within
    # rounding of it
    folder, cfg, w, reqs, _ = models["A", "bfloat16"]
    eng16 = Engine.load(folder, "dtype=bfloat16;max_batch=4;max_tokens=2048")
    near, total = 0, 0
    for p, r in zip(prompts, eng16.generate(prompts, max_tokens=8, stop_ids=[])):
        seq = list(p)
        for tok in r.tokens:
            logits = plain.forward(cfg, w, seq)[-1]
            near += logits.max() - logits[tok] <= TOL_BF16 * np.abs(logits).max()
            total += 1
            seq.append(tok)
    assert total == 8 * len(prompts) and near == total
