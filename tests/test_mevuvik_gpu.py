"""Mevuvik on the GPU against the plain implementation: each mechanism's kernels alone, then whole
models through the trace runner, the step function and the generation entry point, with prompts cut
in every way, batches of unequal requests, reused slots and pages, keys that matter far back and at
page borders, long decoding and the first tokens of a sequence."""
import json
import os

import numpy as np
import pytest
import torch

import plain_mevuvik as plain
from replay_util import Trace, run_trace
from tiny_configs import (MEVUVIK_A, MEVUVIK_B, MEVUVIK_C, _mevuvik_dense, _mevuvik_latent, _mevuvik_moe, _mevuvik_pair)

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


# ------------------------------------------------------------------ mechanisms alone

def _memory_case(rng, n, heads, dim, vdim, extra, planted):
    """Rows [q | k | v | input logits | forget logits | extra columns].  With ``planted``, head 0 forgets
    next to nothing, token 5 writes loudly along its first two channels, every later key is kept off
    them and writes faintly, and the query at token 250 points there."""
    hd, hv = heads * dim, heads * vdim
    x = rng.standard_normal((n, 2 * hd + hv + 2 * heads + extra)) * 0.6
    gates = 2 * hd + hv
    x[:, gates:gates + heads] = rng.standard_normal((n, heads)) * 3.0 - 1.0
    x[:, gates + heads:gates + 2 * heads] = rng.standard_normal((n, heads)) * 2.0 + 2.0
    x[:3, gates:gates + heads] -= 6.0                         # faint first writes: the maximum starts at zero
    if planted:
        x[:, gates + heads] = 30.0
        x[:, gates] = -6.0
        x[5, gates] = 2.0
        x[5, hd:hd + 2] = 4.0
        x[6:, hd:hd + 2] = 0.0
        x[250, :2] = 3.0
        x[250, 2:dim] *= 0.01
        x[5, 2 * hd:2 * hd + vdim] = np.arange(vdim) - 3.0
    return torch.from_numpy(x).float().to(DEV)


@pytest.mark.parametrize("cap", [0.0, 7.0])
@pytest.mark.parametrize("heads,dim,vdim,extra", [(3, 24, 16, 1), (1, 40, 64, 0), (2, 64, 40, 2), (2, 128, 48, 0), (4, 16, 33, 3),
                                                  (1, 200, 8, 0), (2, 33, 20, 1), (1, 256, 17, 3), (5, 8, 5, 0), (2, 32, 16, 0)])
def test_matrix_memory_alone(heads, dim, vdim, extra, cap):
    """Whole sequences against portions of 1, 2, 5, 33 and 17 tokens and token by token (another kernel),
    in slots out of order, twice over in slots that were cleared: S, n and m carry from step to step,
    and the loud write of token 5 is found by the query at token 250 however the walk was cut."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads * 1000 + dim)
    lens, slots = [260, 1, 40, 16], [1, 3, 0, 4]
    hd, hv = heads * dim, heads * vdim
    gates = 2 * hd + hv
    data = [_memory_case(rng, n, heads, dim, vdim, extra, planted=n > 200) for n in lens]
    want, last = [], []
    for x, n in zip(data, lens):
        xn = x.double().cpu().numpy()
        o, state = plain.matrix_memory_scan(xn[:, :hd].reshape(n, heads, dim) * dim ** -0.5, xn[:, hd:2 * hd].reshape(n, heads, dim),
                                            xn[:, 2 * hd:gates].reshape(n, heads, vdim),
                                            plain.capped(xn[:, gates:gates + heads], cap),
                                            plain.log_sigmoid(plain.capped(xn[:, gates + heads:gates + 2 * heads], cap)))
        want.append(o.reshape(n, hv))
        last.append(state)
    # the planted write is what the late query reads
    late = want[0][250, :vdim]
    assert np.corrcoef(late, np.arange(vdim) - 3.0)[0, 1] > 0.9 and np.ptp(late) > 0.5
    state = torch.zeros((6, heads, kernels.matrix_memory_floats(dim, vdim)), dtype=torch.float32, device=DEV)
    aux = torch.zeros((6, heads, kernels.matrix_memory_aux_floats(dim, vdim)), dtype=torch.float32, device=DEV)
    for sizes in ([1000], [1, 2, 5, 33, 17], [1]):
        for s in slots:
            state[s] = 0.0
            aux[s] = 0.0
        got = [np.zeros((n, hv)) for n in lens]
        for live in _steps(lens, sizes):
            x = torch.cat([data[i][lo:hi] for i, lo, hi in live])
            cu, _, slot, _ = _packed([hi - lo for _, lo, hi in live], [slots[i] for i, _, _ in live])
            y = torch.empty((x.shape[0], hv), dtype=torch.float32, device=DEV)
            kernels.matrix_memory(x[:, :hd], x[:, hd:2 * hd], x[:, 2 * hd:gates], x[:, gates:gates + heads],
                                  x[:, gates + heads:gates + 2 * heads], state, aux, cu, slot, y, heads, dim, vdim, cap, dim ** -0.5)
            y = y.double().cpu().numpy()
            at = 0
            for i, lo, hi in live:
                got[i][lo:hi] = y[at:at + hi - lo]
                at += hi - lo
        for i in range(len(lens)):
            # a read-out whose denominator cancels (|n . q| near its floor) is as sensitive as it is large
            assert np.abs(got[i] - want[i]).max() < 1e-4 * max(1.0, np.abs(want[i]).max()), (sizes, i)
            S, n, m = last[i]
            for h in range(heads):
                a = kernels.matrix_memory_matrix(state[slots[i], h], dim, vdim).double().cpu().numpy()
                assert np.abs(a - S[h]).max() < 2e-5 * max(1.0, np.abs(S[h]).max())
                kept = aux[slots[i], h].double().cpu().numpy().reshape(-(-vdim // 16), -1)
                assert np.abs(kept[:, :dim] - n[h]).max() < 2e-5 * max(1.0, np.abs(n[h]).max())
                assert np.abs(kept[:, -4] - m[h]).max() < 2e-5 * max(1.0, abs(m[h]))
        assert not state[2].any() and not state[5].any() and not aux[2].any() and not aux[5].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rd,rot,rank,half", [(3, 24, 12, 12, 44, True), (2, 16, 16, 8, 96, True), (1, 0, 10, 10, 20, True),
                                                        (4, 32, 32, 32, 64, False), (2, 8, 7, 4, 12, True), (2, 8, 0, 0, 16, True)])
def test_latent_rows_and_queries(dtype, heads, dim, rd, rot, rank, half):
    """The kernel between the projections and the attention: the normed latent and the rotated part into
    the page, the queries' parts out, in both layouts of the rotation, also where only the first dims
    turn; sequences that start at positions 0, 61 (a page border inside the step) and 300."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads + rank)
    lens, starts, slots = [7, 9, 1], [0, 61, 300], [1, 0, 2]
    cu, seq, slot, pos = _packed(lens, slots, starts)
    t, base = sum(lens), 700.0
    q, qn = _rand(rng, (t, heads * (dim + rd)))
    kv, kvn = _rand(rng, (t, rank + rd + 5))
    w, wn = _rand(rng, (rank,), shift=1.0, scale=0.2)
    inv = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32, device=DEV) if rot else None
    table = torch.arange(3 * 6, dtype=torch.int32, device=DEV).reshape(3, 6)
    cache = torch.zeros((18, PAGE, rank + rd), dtype=_dt(dtype), device=DEV)
    q_nope = torch.empty((t, heads * dim), dtype=_dt(dtype), device=DEV)
    qa = torch.zeros((t, heads * (rank + rd)), dtype=_dt(dtype), device=DEV)
    dense = torch.empty((t, rank + rd), dtype=_dt(dtype), device=DEV)
    kernels.latent_prepare(q, kv[:, :rank + rd], None, w, 1e-5, inv, rot, 0.3, q_nope, qa, None, cache, table, PAGE, pos, seq, slot,
                           heads, dim, rd, rank, dense=dense, half_layout=half)

    def turned(x):
        if half:
            return plain.rotate_half(x, pos.cpu().numpy(), base, rot)
        order = np.r_[np.arange(0, rot, 2), np.arange(1, rot, 2), np.arange(rot, rd)].astype(int)     # pairs side by side
        y = np.empty_like(x)
        y[..., order] = plain.rotate_half(x[..., order], pos.cpu().numpy(), base, rot)
        return y

    tol = 4e-5 if dtype == "float32" else 1e-2
    qn = qn.reshape(t, heads, dim + rd) * 0.3
    if dim:
        assert np.abs(q_nope.double().cpu().numpy().reshape(t, heads, dim) - qn[..., :dim]).max() < tol * np.abs(qn).max()
    got = qa.double().cpu().numpy().reshape(t, heads, rank + rd)[..., rank:]
    if rd:
        assert np.abs(got - turned(qn[..., dim:])).max() < tol * np.abs(qn).max()
    rows = np.concatenate([plain.rms_norm(kvn[:, :rank], wn, 1e-5), turned(kvn[:, None, rank:rank + rd])[:, 0]], axis=1)
    assert np.abs(dense.double().cpu().numpy() - rows).max() < tol * np.abs(rows).max()
    for i in range(t):
        page = int(table[slots[int(seq[i])], int(pos[i]) // PAGE])
        assert torch.equal(cache[page, int(pos[i]) % PAGE], dense[i])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,n,pad", [(1, 44, 0), (9, 36, 4), (5, 37, 3), (600, 1536, 12), (3, 6000, 0), (2, 6001, 1)])
def test_norms_of_columns_rows_and_embeddings(dtype, rows, n, pad):
    """The norm of a slice of columns; a row added to every row with the norm that follows; a table's rows
    normed: widths that are and are no multiple of four, short rows and rows read twice."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(n)
    wide, widen = _rand(rng, (rows, n + pad), scale=2.0)
    w, wn = _rand(rng, (n,), shift=1.0, scale=0.3)
    tol = 1e-5 if dtype == "float32" else 1e-2

    def close(got, want):
        assert np.abs(got.double().cpu().numpy() - want).max() < tol * np.abs(want).max()

    out = torch.empty((rows, n), dtype=_dt(dtype), device=DEV)
    kernels.norm_cols(wide[:, pad:], w, out, 1e-4)
    close(out, plain.rms_norm(widen[:, pad:], wn, 1e-4))
    x, xn = _rand(rng, (rows, n), scale=2.0)
    v, vn = _rand(rng, (n,))
    kernels.add_row(v, x, (w, 1e-4, out))
    close(out, plain.rms_norm(xn + vn, wn, 1e-4))
    assert np.abs(x.double().cpu().numpy() - (xn + vn)).max() < 1e-6 * np.abs(xn).max()
    kernels.add_row(v, x)
    assert np.abs(x.double().cpu().numpy() - (xn + 2 * vn)).max() < 1e-6 * np.abs(xn).max()
    table, tablen = _rand(rng, (11, n), _dt(dtype))
    ids = rng.integers(0, 11, rows)
    x = torch.empty((rows, n), dtype=torch.float32, device=DEV)
    kernels.embed_norm(table, _i32(ids), w, x, 1.5, 1e-4)
    assert np.abs(x.double().cpu().numpy() - plain.rms_norm(tablen[ids] * 1.5, wn, 1e-4)).max() < 1e-5 * 5
    logits, logitsn = _rand(rng, (rows, n), scale=20.0)
    kernels.cap_rows(logits, 9.0)
    assert np.abs(logits.double().cpu().numpy() - plain.capped(logitsn, 9.0)).max() < 1e-5 * 9


@pytest.mark.parametrize("m,n,k", [(1, 200, 72), (1, 512, 2048), (7, 96, 128), (8, 384, 1024), (20, 130, 64), (33, 256, 2560),
                                   (64, 72, 512), (65, 200, 128), (130, 320, 96), (300, 520, 200), (700, 1024, 320), (5, 50, 52)])
def test_product_with_an_activation_and_with_a_factor_per_feature(m, n, k):
    """Every way a product takes (plain, one tile, the inner dimension split over a cluster, persistent with
    and without a cut last round): act(x W^T + b) in the result's type, and y += s * (x W^T + b)."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(m + n + k)
    for dtype in ("float32", "bfloat16"):
        x, xn = _rand(rng, (m, k), _dt(dtype))
        w, wn = _rand(rng, (n, k), _dt(dtype), scale=k ** -0.5)
        b, bn = _rand(rng, (n,))
        s, sn = _rand(rng, (n,), shift=0.5)
        r, rn = _rand(rng, (m, n), scale=2.0)
        z = xn @ wn.T + bn
        tol = 3e-5 if dtype == "float32" else 1.2e-2
        for act, fn in (("relu2", plain.relu_squared), ("gelu", None)):
            out = torch.empty((m, n), dtype=_dt(dtype), device=DEV)
            kernels.gemm(x, w, out, b, act=act)
            want = fn(z) if fn else torch.nn.functional.gelu(torch.from_numpy(z)).numpy()
            assert np.abs(out.double().cpu().numpy() - want).max() < tol * np.abs(want).max(), (dtype, act)
        kernels.gemm(x, w, r, b, accumulate=True, col_scale=s)
        want = rn + sn * z
        assert np.abs(r.double().cpu().numpy() - want).max() < 3e-5 * np.abs(want).max(), dtype
    kernels.check_status()


def test_a_factor_per_feature_before_the_norm_that_follows():
    """Decode steps: the product that adds into the stream leaves the next norm's input; the factor is in it."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(4)
    for m, n, k in ((1, 512, 2048), (8, 320, 1024), (40, 640, 1536)):
        x, xn = _rand(rng, (m, k), torch.bfloat16)
        w, wn = _rand(rng, (n, k), torch.bfloat16, scale=k ** -0.5)
        s, sn = _rand(rng, (n,), shift=0.5)
        g, gn = _rand(rng, (n,), shift=1.0, scale=0.2)
        r, rn = _rand(rng, (m, n), scale=2.0)
        left = kernels.gemm(x, w, r, accumulate=True, then_norm=(g, 1e-5), col_scale=s)
        assert left is not None
        new = rn + sn * (xn @ wn.T)
        assert np.abs(r.double().cpu().numpy() - new).max() < 3e-5 * np.abs(new).max()
        want = plain.rms_norm(new, gn, 1e-5)
        assert np.abs(left.materialize().double().cpu().numpy() - want).max() < 1e-2 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("t,width,experts,top,ff", [(1, 64, 4, 2, 32), (9, 52, 3, 3, 20), (15, 72, 6, 1, 40), (40, 64, 5, 2, 48),
                                                    (255, 128, 16, 4, 64), (300, 128, 9, 3, 64), (700, 64, 4, 4, 32)])
def test_sigmoid_routing_and_squared_relu_experts(dtype, t, width, experts, top, ff):
    """Token-major (fewer than 16 tokens, and float32), grouped (16 to 255) and on the tcgen05 product
    (256 and more), with a factor per feature on what is added.  The correction turns some choices around."""
    from gemmars_b200.parts.base import build_part
    from gemmars_b200.parts.plan import PartSpec
    rng = np.random.default_rng(t + experts)
    names, w, wn = {}, {}, {}

    def add(name, short, shape, scale, dt=torch.bfloat16):
        names[short] = name
        w[short], wn[name] = _rand(rng, shape, dt, scale=scale)

    add("router", "router", (experts, width), 0.4)
    add("correction", "router_bias", (experts,), 0.3, torch.float32)
    for e in range(experts):
        add(f"e{e}.up", f"e{e}.up", (ff, width), 0.25)
        add(f"e{e}.down", f"e{e}.down", (width, ff), 0.1)
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": 1.7}, "expert": {"ff": ff}}
    part = build_part("ffn", PartSpec("moe", {"hidden_size": width, "experts": experts, "top": top, "ff": ff, "limit": None,
                                              "router_bias": True, "gated": False, "activation": "relu2", "routing": "sigmoid",
                                              "routing_scale": 1.7, "shared": None}, names), dtype)
    part.load({k: v if k == "router_bias" else v.to(_dt(dtype)) for k, v in w.items()})
    s, sn = _rand(rng, (width,), shift=0.8)
    part.set_output_scale(s)
    h, hn = _rand(rng, (t, width), _dt(dtype))
    res, resn = _rand(rng, (t, width), torch.float32)
    part.forward(type("Ctx", (), dict(host=None))(), h, res)
    want = resn + sn * plain.routed_ffn(hn, wn, mlp)
    # a token whose last chosen and first unchosen scores are closer than rounding may go either way
    z = hn @ wn["router"].T
    if top < experts and t > 30:
        order = lambda a: np.argsort(-a, axis=1)[:, :top]                                   # noqa: E731
        turned = (np.sort(order(z)) != np.sort(order(plain.sigmoid(z) + wn["correction"]))).any(axis=1)
        assert turned.any()                                                                 # the correction matters
    c = np.sort(plain.sigmoid(z) + wn["correction"], axis=1)[:, ::-1]
    sure = np.ones(t, bool) if top == experts else (c[:, top - 1] - c[:, top]) > (1e-5 if dtype == "float32" else 0.01)
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    assert sure.mean() > 0.6
    assert np.abs(res.double().cpu().numpy() - want)[sure].max() <= tol * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,groups,dim,vdim,new", [(3, 1, 16, 24, 70), (3, 1, 16, 24, 1), (8, 2, 64, 40, 33), (8, 2, 64, 40, 1),
                                                       (5, 5, 20, 12, 9), (5, 5, 20, 12, 1)])
def test_one_gate_per_head_on_the_attention(dtype, heads, groups, dim, vdim, new):
    """Prompts and single tokens, on the tensor cores and on the plain kernel; an odd number of heads; a
    query that points at one key far back across a page border."""
    from gemmars_b200 import kernels
    rng = np.random.default_rng(heads + new)
    total, dt = 130, _dt(dtype)
    q, qn = _rand(rng, (new, heads * dim), dt)
    k, kn = _rand(rng, (total, groups, dim), dt, scale=0.3)
    v, vn = _rand(rng, (total, groups, vdim), dt)
    g, gn = _rand(rng, (new, heads + 3), dt, scale=2.0)
    far = total - new if new > 1 else 63
    with torch.no_grad():
        q[-1, :dim] = 0.0
        q[-1, 0] = 8.0
        k[far, 0] = 0.0
        k[far, 0, 0] = 8.0                                 # one score of 64 times the scale stands out
    qn, kn = q.double().cpu().numpy(), k.double().cpu().numpy()
    table = _i32([[4, 2, 3]])
    kc = torch.zeros((5, groups, PAGE, dim), dtype=dt, device=DEV)
    vc = torch.zeros((5, groups, vdim, PAGE), dtype=dt, device=DEV)
    for p in range(total):
        page = int(table[0, p // PAGE])
        kc[page, :, p % PAGE], vc[page, :, :, p % PAGE] = k[p], v[p]
    cu, seq, slot, pos = _packed([new], [0], [total - new])
    ctx = type("Ctx", (), dict(cu_seqlens=cu, seq_start=_i32([total - new]), seq_slot=slot, n_seqs=1, tok_pos=pos, tok_seq=seq))()
    out = torch.empty((new, heads * vdim), dtype=dt, device=DEV)
    kernels.attention_capped(ctx, q, out, heads, kc, vc, table, PAGE, None, 0.25, 0.0, g[:, 2:], 1.3, gate_per_head=True)
    full = plain.causal_attention(np.concatenate([np.zeros((total - new, heads, dim)), qn.reshape(new, heads, dim)]), kn, vn, 0.25)
    want = 1.3 * full[total - new:] * plain.sigmoid(gn[:, 2:2 + heads])[:, :, None]
    assert np.abs(want[-1, 0] / 1.3 / plain.sigmoid(gn[-1, 2]) - vn[far, 0]).max() < 0.01
    assert np.abs(out.double().cpu().numpy().reshape(new, heads, vdim) - want).max() < (2e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()


# ------------------------------------------------------------------ whole models

def _sharp_folder(tmp_path_factory, raw, seed, factor):
    """Random weights whose attention queries and keys are scaled by ``factor``: scores grow with its
    square, the softmax picks single keys instead of averaging, and a wrong key, page, slot or rotation
    shows in the logits.  The gates of the memories are spread, so that single writes stand out, and the
    vectors of the passes are loud."""
    from gemmars_b200.weights import random_weights, write_safetensors
    tensors = random_weights(raw, seed=seed)
    for name in tensors:
        if name.endswith((".mix.uq", ".left.q", ".left.k", ".mix.uk", ".mix.dkv")):
            tensors[name] = (tensors[name].float() * factor).bfloat16()
        elif name.endswith((".right.i", ".right.f", ".right.q")):
            tensors[name] = (tensors[name].float() * 12.0).bfloat16()
        elif name == "loop.step":
            tensors[name] = (tensors[name].float() * 10.0).bfloat16()
        elif name.endswith((".right.o", ".mix.o", ".left.o")):
            tensors[name] = (tensors[name].float() * (30.0 if ".left." in name else 14.0)).bfloat16()
        elif name.endswith(".up"):
            tensors[name] = (tensors[name].float() * 4.0).bfloat16()
        elif name.endswith((".correction", ".mlp.router")):
            tensors[name] = (tensors[name].float() * (2.0 if name.endswith("correction") else 6.0)).bfloat16()
        elif name == "head":
            tensors[name] = (tensors[name].float() * 12.0).bfloat16()
    d = str(tmp_path_factory.mktemp("mevuvik"))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(raw, f)
    write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d


def _within(errors, tol, dtype, what, share=0.04):
    """float32: every position within ``tol``.  bfloat16: rounding the router's input moves a token
    whose candidate experts have nearly equal scores to another expert now and then, which changes
    that position's logits (and through the states, a few after it) by more than rounding; up to
    ``share`` of the positions (at least one) may be over, and the rest must be within ``tol``."""
    errors = np.asarray(errors)
    over = int((errors > tol).sum())
    allowed = 0 if dtype == "float32" else max(1, int(share * errors.size))
    assert over <= allowed, f"{what}: {over} of {errors.size} positions are over {tol:.2e} (worst {errors.max():.2e})"


REQUESTS = {"A": (MEVUVIK_A, [15, 21, 9, 70, 44, 131]), "B": (MEVUVIK_B, [17, 33, 3, 80, 150, 300])}
GROUPS = [[0, 1, 2], [3, 4, 5]]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (raw, lengths) in REQUESTS.items():
        folder = _sharp_folder(tmp_path_factory, raw, seed=31 + len(name), factor=11.0 if name == "A" else 6.0)
        cfg, w = plain.load_folder(folder)
        rng = np.random.default_rng(lengths[0])
        reqs = [rng.integers(0, raw["vocab"], n).tolist() for n in lengths]
        out[name] = (folder, cfg, w, reqs, [plain.forward(cfg, w, r) for r in reqs])
    return out


def test_the_test_models_show_a_fault(models):
    """The scaled weights do what they are for: in the plain model, queries rotated one position too far, a
    lost first key, a lost head gate, a memory that forgets a little faster, a read-out without the
    floor of its denominator, one pass's vector for all passes, a choice without the correction, or the
    relu without its square move the logits by far more than any tolerance."""
    folder, cfg, w, reqs, ref = models["A"]
    toks = reqs[5]
    scale = np.abs(ref[5]).max()

    def planted(name, fault):
        saved = getattr(plain, name)
        try:
            setattr(plain, name, fault(saved))
            return plain.forward(cfg, w, toks)
        finally:
            setattr(plain, name, saved)

    def head_gate(inner):
        return lambda h, P, m: inner(h, {**P, "g": np.zeros_like(P["g"])}, m)

    def floor(inner):
        def scan(q, k, v, i, f, state=None):
            return inner(q, k, v, i + 40.0, f)            # the same memory times e^40: its floor of one is out of reach
        return scan

    def drift(inner):
        def scan(q, k, v, i, f, state=None):
            return inner(q, k, v, i, f - 0.1)
        return scan

    runs = {"rotation": planted("rotate_half", lambda f: lambda x, pos, base, dims: f(x, np.asarray(pos) + (x.shape[1] > 1), base, dims)),
            "first key": planted("causal_attention", lambda f: lambda q, k, v, s: f(q, np.concatenate([0 * k[:1], k[1:]]), v, s)),
            "head gate": planted("head_gated_attention_mixer", head_gate), "floor": planted("matrix_memory_scan", floor),
            "forgetting": planted("matrix_memory_scan", drift),
            "correction": planted("route_sigmoid", lambda f: lambda z, c, top, s: f(z, 0 * c, top, s)),
            "relu": planted("relu_squared", lambda f: lambda z: np.maximum(z, 0.0)),
            "pass": plain.forward(cfg, {**w, "loop.step": np.vstack([w["loop.step"][0]] * 2)}, toks)}
    for what, other in runs.items():
        moved = np.abs(other - ref[5]).max(axis=1)
        assert moved.max() > 2 * TOL_BF16 * scale and (moved[40:] > 100 * TOL_F32 * scale).mean() > 0.3, (what, moved.max() / scale)


@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_all_cuttings_match_the_plain_implementation(name, dtype, models, tmp_path):
    """Through bin/trace_run: each request whole, with its last 40 tokens one by one, and in two batches of
    unequal requests that follow one another in a cache sized to the peak, so that the second batch
    lives in the slots and pages the first gave back."""
    folder, cfg, w, reqs, ref = models[name]
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
        _within([np.abs(got[(f"{tag}{i}", p)] - r[p]).max() for i, r in enumerate(ref) for p in range(len(r))], tol, dtype,
                f"cutting {tag!r}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_after_every_run_of_a_layer(dtype, models):
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, _ = models["A"]
    toks = reqs[3]
    _, want = plain.forward(cfg, w, toks, return_layers=True)
    model = build_model(folder, dtype=dtype)
    assert len(model.blocks) == 4 and len(model.plan.schedule) == 6 == len(want)
    seen = []
    for block in model.blocks:
        def run(ctx, x, caches, _inner=block.forward, **kw):
            left = _inner(ctx, x, caches, **kw)
            assert x.dtype == torch.float32                      # the residual stream is 32-bit in both modes
            seen.append(x.double().cpu().numpy())
            return left
        block.forward = run
    runner = Runner(model, max_tokens=256, max_batch=1, use_graphs=False)
    runner.step([StepItem(runner.open(), toks, [])])
    assert len(seen) == len(want)
    for i, (a, b) in enumerate(zip(seen, want)):
        tol = (1e-5 if dtype == "float32" else 2e-2) * np.abs(b).max()
        # the stream itself, not logits: a token that went to another expert early stays off through every layer
        _within(np.abs(a - b).max(axis=1), tol, dtype, f"run {i}", share=0.08)


@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_long_decoding_and_reused_slots(name, dtype, models):
    """One runner, a cache of eight pages.  A prompt in portions of 2, 3, 64, 1, 65 and the rest;
    another from its first token one by one for 300 steps, across four page borders, beside a neighbour
    that comes and goes; then the same again in the slots and pages given back: in float32 to the last bit."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, ref = models[name]
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
        _within([np.abs(got[("a", p)] - ref[4][p]).max() for p in range(len(reqs[4]))], tol, dtype, "portions")
        _within([np.abs(got[("b", p)] - long_ref[p]).max() for p in range(len(long_toks))], tol, dtype, "decoded")
        _within([np.abs(got[("c", p)] - ref[0][p]).max() for p in range(len(reqs[0]))], tol, dtype, "neighbour")
        if first_round is None:
            first_round = got
        elif dtype == "float32":
            assert all(np.array_equal(got[k], first_round[k]) for k in got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_the_tensor_cores_do_not_take(dtype, tmp_path_factory):
    """A width of 52 and heads of 20, 12, 9, 7 and 5: every product and the attention run on the plain
    kernels; no loop, no cap.  Prompts in portions of two tokens, then token by token, against the whole."""
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder = _sharp_folder(tmp_path_factory, MEVUVIK_C, seed=5, factor=10.0)
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
    _within(errs, (TOL_F32 if dtype == "float32" else TOL_BF16) * scale, dtype, "portions of two")
    for s in slots:
        runner.close(s)
    assert runner.cache.pages_held() == 0


def test_long_prompts_on_the_tensor_cores(models):
    """Prompts of more than 256 tokens: keys and values expanded per head, experts on the tcgen05 product;
    one alone, two in one step, one in two portions (the second reads the latent rows of the first)."""
    from gemmars_b200 import kernels
    from gemmars_b200.engine import Runner, StepItem, build_model
    folder, cfg, w, reqs, _ = models["B"]
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
    _within(errs, TOL_BF16 * scale, "bfloat16", "long prompts")


def _random_configuration(rng):
    """Layers of both kinds in any order with sizes drawn at random, some of them in a loop."""
    def mlp():
        r = rng.random()
        if r < 0.15:
            return None
        if r < 0.5:
            return _mevuvik_dense(int(rng.choice([24, 52, 96, 130])))
        experts = int(rng.integers(1, 13))
        return _mevuvik_moe(experts, int(rng.integers(1, min(experts, 6) + 1)), int(rng.choice([24, 32, 40, 66])), float(rng.uniform(0.5, 3.0)))

    def latent():
        dim, rd = int(rng.choice([4, 16, 24, 32, 64])), int(rng.choice([2, 8, 16, 20, 32]))
        return _mevuvik_latent(int(rng.integers(1, 7)), dim, rd, int(rng.choice([8, 16, 20, 32, 48])), int(rng.choice([10, 24, 48, 96])),
                               int(rng.choice([12, 32, 48, 80, 160])), float((dim + rd) ** -0.5 * rng.uniform(0.7, 1.5)),
                               float(rng.choice([1e4, 3e5, 100.0])))

    def pair():
        g = int(rng.choice([1, 2, 3]))
        d = int(rng.choice([12, 16, 32, 64, 80]))
        left = (g * int(rng.choice([1, 2, 3])), g, d, int(rng.choice([16, 40, 64, d])), float(d ** -0.5 * rng.uniform(0.7, 1.5)))
        right = (int(rng.integers(1, 7)), int(rng.choice([6, 16, 24, 48, 64, 72, 130])), int(rng.choice([10, 16, 40, 64])),
                 float(rng.choice([1.0, 4.0, 15.0])))
        return _mevuvik_pair(left, right, float(rng.uniform(0.3, 1.2)), float(rng.uniform(0.3, 1.2)))

    n = int(rng.integers(1, 6))
    layers = []
    for _ in range(n):
        kind = str(rng.choice(["latent_attention", "parallel"]))
        layers.append({"type": kind, "mixer": latent() if kind == "latent_attention" else pair(), "mlp": mlp()})
    out = {"architecture": "Mevuvik", "vocab": int(rng.choice([97, 300, 1000])), "width": int(rng.choice([52, 64, 96, 136, 200])),
           "norm": {"eps": float(rng.choice([1e-5, 1e-6]))}, "residual_mult": float(rng.choice([1.0, 0.5, 0.22])),
           "logit_softcap": float(rng.choice([5.0, 30.0])) if rng.random() < 0.8 else None, "layers": layers}
    if rng.random() < 0.8:
        start = int(rng.integers(0, n))
        out["loop"] = {"start": start, "stop": int(rng.integers(start + 1, n + 1)), "times": int(rng.integers(1, 4))}
    return out


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
        out = runner.step([StepItem(slots[i], [reqs[i][heads[i] + k]], [0]) for i in live]).cpu().numpy()
        errs += [np.abs(out[n] - ref[i][heads[i] + k]).max() for n, i in enumerate(live)]
    assert len(errs) == sum(lens)
    assert max(errs) <= TOL_F32 * scale, f"{max(errs) / scale:.2e} of the largest logit, configuration {json.dumps(raw)}"
    for s in slots:
        runner.close(s)
    assert runner.cache.pages_held() == 0


def test_greedy_generation_through_the_engine(models):
    from gemmars_b200 import Engine
    folder, cfg, w, reqs, _ = models["A"]
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
    # rounding of it (but for the few that follow a token routed to another expert, see _within)
    eng16 = Engine.load(folder, "dtype=bfloat16;max_batch=4;max_tokens=2048")
    near, total = 0, 0
    for p, r in zip(prompts, eng16.generate(prompts, max_tokens=8, stop_ids=[])):
        seq = list(p)
        for tok in r.tokens:
            logits = plain.forward(cfg, w, seq)[-1]
            near += logits.max() - logits[tok] <= TOL_BF16 * np.abs(logits).max()
            total += 1
            seq.append(tok)
    assert total == 8 * len(prompts) and near >= 0.9 * total
