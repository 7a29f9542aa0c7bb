"""Padulorn through the framework (kernels, page pool and state slots, ragged steps, scheduler) against the plain oracle
(oracle/padulorn_oracle.py): every mechanism alone, then whole models under every way of cutting and batching the work."""
import json
import os
import struct
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from oracle import padulorn_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 1e-4, 4e-2
F32, BF16 = torch.float32, torch.bfloat16


def attention(heads=4, kv_heads=2, dim=24, vdim=20, size=37, keep_first=5, rot_dims=12, base=900.0, scaling=(6.0, 64, 9.0, 1.0), v_mix=True, scale=None):
    rot = {"base": base, "dims": rot_dims} if rot_dims else None
    if rot and scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=rot, scale=scale if scale is not None else dim ** -0.5,
                                               mask={"size": size, "keep_first": keep_first} if size else None, v_mix=v_mix)}


def retention(heads=3, dim=16, vdim=24, decay=None, rot_dims=8, base=700.0):
    decay = decay if decay is not None else [1.0 - 2.0 ** (-1.5 - 2.3 * h) for h in range(heads)]
    return {"type": "retention", "mixer": dict(heads=heads, dim=dim, vdim=vdim, decay=decay, rot={"base": base, "dims": rot_dims} if rot_dims else None)}


def moe(l, experts=8, top=3, ff=40, groups=(4, 2)):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return dict(l, mlp={"kind": "moe", "expert": {"ff": ff}, "router": router})


def bare(l):
    return dict(l, mlp=None)


def make_cfg(layers, width=72, vocab=90, eps=1e-5, embed=5.0, mult=0.8, logit=0.7):
    return {"architecture": "Padulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed}, "residual_mult": mult, "logit_scale": logit,
            "layers": layers}


# both mixers twice, the blending source not the first layer, a layer without feed-forward, a full-context layer, unequal windows
BASE_CFG = make_cfg([moe(retention()), moe(attention()), bare(retention(heads=2, dim=24, vdim=16, rot_dims=24)), moe(attention(size=None, v_mix=False, rot_dims=24, scaling=None), 6, 2, 33, None),
                     moe(attention(heads=2, kv_heads=2, size=64, keep_first=1), 9, 1, 24, (3, 1))])


def build(cfg, w, dtype):
    from paligemma_multimodal_system_b200.modeling_padulorn import PadulornConfig, PadulornForCausalLM
    return PadulornForCausalLM(PadulornConfig(cfg), dtype).load_weights({k: v.to(BF16) for k, v in w.items()})


def engine_for(cfg, w, dtype, max_tokens=1024, slots=4):
    from paligemma_multimodal_system_b200.engine import SequenceEngine
    return SequenceEngine(build(cfg, w, dtype), max_tokens, slots)


def poison(engine):
    """Stale memory must never be read: pages and state slots start as huge values instead of zeros."""
    for t in engine.store.k_pages + engine.store.v_pages + engine.store.state:
        if t is not None:
            t.fill_(1e4)


def rows_of(t, n):
    return t.double().cpu().reshape(n, -1)


def worst_row(got, ref):
    """The largest error of any row, relative to the typical row's size (one wrong position must not drown among hundreds)."""
    got, ref = rows_of(got, ref.shape[0]), rows_of(ref, ref.shape[0])
    return float(((got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()).max())


def median_row(got, ref):
    got, ref = rows_of(got, ref.shape[0]), rows_of(ref, ref.shape[0])
    return float(((got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()).median())


def close(got, ref, dtype):
    """fp32: every row within F32_TOL.  bf16: half the rows within BF16_TOL / 2 and no row beyond twice BF16_TOL."""
    if dtype == F32:
        return worst_row(got, ref) < F32_TOL
    return median_row(got, ref) < BF16_TOL / 2 and worst_row(got, ref) < 2 * BF16_TOL


def margins(z, router):
    """How decided each row's choice of experts is: the smallest gap between what is taken and what is left (groups, then experts)."""
    s, n, top = torch.sigmoid(z), z.shape[1], router["top"]
    gap = torch.full((z.shape[0],), 9.0)
    groups = router.get("groups")
    if groups and groups["keep"] < groups["count"]:
        per = s.view(-1, groups["count"], n // groups["count"])
        score = per.topk(min(2, per.shape[2]), -1).values.sum(-1)
        best = score.topk(groups["keep"] + 1, -1)
        gap = best.values[:, -2] - best.values[:, -1]
        kept = torch.zeros_like(score).scatter_(1, best.indices[:, :-1], 1.0).bool()
        s = torch.where(kept[:, :, None], per, torch.full_like(per, -9.0)).reshape(-1, n)
    if top < n:
        t = s.topk(top + 1, -1).values
        gap = torch.minimum(gap, t[:, -2] - t[:, -1])
    return gap


def steady_weights(cfg, seed):
    """Random weights under which bf16 rounding cannot tip a choice of experts: the routers read a few columns of the residual that no
    sub-layer writes (zero norm weights there), so a token's choice is its embedding's, and embeddings with close calls are drawn again."""
    w, R = O.random_weights(cfg, seed), 6
    g = torch.Generator().manual_seed(seed)
    emb, scale, routed = w["embed"], cfg["embedding"]["scale"], []
    for i, l in enumerate(cfg["layers"]):
        w[f"l{i}.norm1"][-R:] = 0.0
        if l.get("mlp"):
            w[f"l{i}.norm2"][-R:] = 0.0
            r = w[f"l{i}.mlp.router"]
            r[:, :-R], r[:, -R:] = 0.0, (0.6 * torch.randn(r.shape[0], R, generator=g)).to(BF16).float()
            routed.append((r[:, -R:], l["mlp"]["router"]))
    for _ in range(300):
        close_calls = torch.zeros(emb.shape[0], dtype=torch.bool)
        for r, router in routed:
            close_calls |= margins(scale * emb[:, -R:] @ r.T, router) < 0.015
        if not bool(close_calls.any()):
            return w
        emb[close_calls, -R:] = (torch.randn(int(close_calls.sum()), R, generator=g) / scale).to(BF16).float()
    raise AssertionError("no decided embeddings found")


def toks(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def run_cut(engine, rid, tokens, cuts):
    """Feeds `tokens` in portions of the given sizes (the last size repeats); returns logits of every position."""
    out, pos, i = [], 0, 0
    while pos < len(tokens):
        k = min(cuts[min(i, len(cuts) - 1)], len(tokens) - pos)
        out.append(engine.step([(rid, tokens[pos:pos + k], list(range(k)))], [rid] if pos + k == len(tokens) else []))
        pos, i = pos + k, i + 1
    return torch.cat(out)


def one_store(layout, T, dtype, skip_pages=2):
    """A store with one admitted sequence of up to T tokens whose pages do not start at page 0 and whose slot is not slot 0."""
    from paligemma_multimodal_system_b200.cache import SequenceStore
    store = SequenceStore(layout, max_tokens=(T + 63) // 64 * 64 + 64 * skip_pages, num_slots=2, dtype=dtype)
    store.pool.take(skip_pages)
    store.admit("skipped")
    store.admit(0)
    store.reserve(0, T)
    for t in store.k_pages + store.v_pages + store.state:
        if t is not None:
            t.fill_(1e4)
    return store


def run_mixer(mx, h, cuts, dtype, prec, first_values=None):
    """h [T, D] through a mixer in portions; returns fp32 [T, D] on the CPU."""
    from paligemma_multimodal_system_b200 import seq_ops
    T = h.shape[0]
    store = one_store(mx.cache_specs(), T, dtype)
    rec, pos, outs, i = store.live[0], 0, [], 0
    while pos < T:
        k = min(cuts[min(i, len(cuts) - 1)], T - pos)
        b = seq_ops.step_scope(seq_ops.make_step_batch([dict(tokens=[0] * k, ctx=pos, slot=rec.slot, pages=rec.pages)]))
        if first_values is not None:
            b.shared["values"] = first_values[pos:pos + k].cuda().to(dtype)
        outs.append(mx(h[pos:pos + k].cuda().to(dtype).contiguous(), b, store, 0, prec).float().cpu())
        pos, i = pos + k, i + 1
    return torch.cat(outs)


def load_mixer(cfg, w, i=0):
    from paligemma_multimodal_system_b200.modeling_padulorn import PadulornConfig, _mixer
    mx = _mixer(PadulornConfig(cfg), i)
    left = {k: v.to(BF16) for k, v in w.items()}
    mx.load(lambda name, shape: left.pop(name), f"l{i}.mix.")
    return mx


def ragged(lens, plans):
    """Steps of several sequences in unequal portions: yields (rows of the step as (sequence, first, count), batch)."""
    from paligemma_multimodal_system_b200 import seq_ops
    fed = [0] * len(lens)
    for step in range(max(map(len, plans))):
        rows, es = [], []
        for i, plan in enumerate(plans):
            if step < len(plan) and plan[step]:
                k = plan[step]
                es.append(dict(tokens=[0] * k, ctx=fed[i], slot=len(lens) - i, pages=list(range((fed[i] + k + 63) // 64))))
                rows.append((i, fed[i], k))
                fed[i] += k
        yield rows, seq_ops.make_step_batch(es)
    assert fed == lens


# ----------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ----------------------------------------------------------------------------------------------------------------------
LENS = [143, 9, 66]
PLANS = [[5, 1, 2, 75, 60], [1] * 9, [2, 2, 15, 16, 31]]
BLOCK_PLANS = [[143], [9], [16, 33, 17]]
HEADS = [(4, 24, 20, 12), (3, 64, 64, 64), (2, 48, 128, 16), (2, 128, 72, 128), (5, 7, 9, 4), (1, 100, 33, 50), (2, 200, 16, 8), (2, 96, 48, 0), (3, 32, 8, 32), (1, 1, 1, 0), (2, 256, 24, 256)]


@pytest.mark.parametrize("H,dim,vdim,rot", HEADS)
@pytest.mark.parametrize("f32,plans,blocks", [(True, PLANS, None), (True, PLANS, True), (False, PLANS, None), (False, BLOCK_PLANS, None), (False, PLANS, True), (False, PLANS, False)])
def test_retention_recurrence(H, dim, vdim, rot, f32, plans, blocks):
    """Scan and both block kernels (entries shorter than, equal to and longer than a block) against the recurrence; decays of exactly one,
    slow, fast and nearly zero; slots full of garbage at the start."""
    from paligemma_multimodal_system_b200 import seq_ops
    from paligemma_multimodal_system_b200.mixers import rotary_frequencies
    dt = F32 if f32 else BF16
    g = torch.Generator().manual_seed(dim * vdim)
    decay = torch.tensor([1.0, 0.97, 0.5, 1e-3, 0.9995])[:H]
    kscale, base = 0.3, 60.0
    W = H * (2 * dim + vdim)
    data = [torch.randn(n, (W + 7) // 8 * 8, generator=g).to(BF16).float() for n in LENS]
    ref = []
    for x in data:
        n = x.shape[0]
        q, k, v = (t.double().view(n, H, -1) for t in torch.split(x[:, :W], [H * dim, H * dim, H * vdim], 1))
        r = {"base": base, "dims": rot}
        q = torch.stack([O.turned(q[t], t, r, "next") for t in range(n)])
        k = torch.stack([O.turned(k[t], t, r, "next") for t in range(n)]) * kscale
        ref.append(O.retained(q, k, v, decay.double()))
    state = torch.full((4, H, dim, vdim), 1e4, device="cuda")
    freq = rotary_frequencies(base, rot).cuda() if rot else None
    got = [[] for _ in LENS]
    for rows, b in ragged(LENS, plans):
        x = torch.cat([data[i][p:p + k] for i, p, k in rows]).cuda().to(dt)
        out = torch.full((b.T, H * vdim), float("nan"), device="cuda")
        turn = seq_ops.rotary_table(b, freq, rot, dim) if rot else None
        seq_ops.retention(x, state, decay.cuda(), out, b, H, dim, vdim, kscale=kscale, rotate=turn, blocks=blocks)
        r = 0
        for i, _, k in rows:
            got[i].append(out[r:r + k].cpu())
            r += k
    for i in range(3):
        y = torch.cat(got[i]).view(-1, H, vdim)
        for h in range(H):  # head by head: a slow head's large values must not hide a fast one's
            assert worst_row(y[:, h], ref[i][:, h]) < 2e-5, (i, h)


def test_a_token_written_long_ago_is_read_back_from_the_state():
    """One token's key is a direction no other key has; hundreds of tokens later a query along it must return that token's value times the
    decay's power, across portion, block and form borders."""
    from paligemma_multimodal_system_b200 import seq_ops
    H, dim, vdim, n = 2, 16, 24, 400
    g = torch.Generator().manual_seed(0)
    decay = torch.tensor([1.0, 0.995])
    for mark in (0, 15, 16, 17, 63, 64, 99):
        k = torch.randn(n, H, dim, generator=g)
        k[..., 0] = 0.0
        k[mark] = 0.0
        k[mark, :, 0] = 1.0
        v, q = torch.randn(n, H, vdim, generator=g), torch.zeros(n, H, dim)
        q[..., 0] = 1.0
        x = torch.cat([t.reshape(n, -1) for t in (q, k, v)], 1).to(BF16)
        want = x[mark, -H * vdim:].double().view(H, vdim) * decay.double()[:, None] ** (n - 1 - mark)
        for dt in (F32, BF16):
            for cuts in ([n], [mark + 1, 1], [100, 2, 298], [70, 15]):
                state = torch.full((1, H, dim, vdim), 1e4, device="cuda")
                pos, i, last = 0, 0, None
                while pos < n:
                    c = min(cuts[min(i, len(cuts) - 1)], n - pos)
                    b = seq_ops.make_step_batch([dict(tokens=[0] * c, ctx=pos, slot=0, pages=list(range((pos + c + 63) // 64)))])
                    out = torch.empty(c, H * vdim, device="cuda")
                    seq_ops.retention(x[pos:pos + c].cuda().to(dt).contiguous(), state, decay.cuda(), out, b, H, dim, vdim)
                    last, pos, i = out[-1].cpu(), pos + c, i + 1
                assert worst_row(last.view(H, vdim), want) < 1e-4, (mark, dt, cuts)


@pytest.mark.parametrize("rows,groups,size", [(5, 4, 24), (1, 1, 130), (33, 3, 7), (8, 16, 64), (3, 2, 1024), (2, 40, 6), (4, 1, 1)])
@pytest.mark.parametrize("f32", [True, False])
def test_head_norm_without_weight_and_silu_gate(rows, groups, size, f32):
    from paligemma_multimodal_system_b200 import seq_ops
    dt, D, eps = (F32 if f32 else BF16), groups * size, 1e-3
    g = torch.Generator().manual_seed(D)
    o, gate = 0.05 * torch.randn(rows, D, generator=g), torch.randn(rows, D, generator=g).to(BF16).float()
    buf = torch.full((rows, D + 8), 3.0, device="cuda", dtype=dt)
    seq_ops.group_norm_gate(o.cuda(), None, gate.cuda().to(dt), buf[:, :D], groups, eps, seq_ops.GATE_SILU_AFTER, 0.7)
    assert worst_row(buf[:, :D].float(), 0.7 * O.over_rms(o.view(rows, groups, size), eps).reshape(rows, D) * O.silu(gate)) < (1e-5 if f32 else 1e-2)
    seq_ops.group_norm_gate(o.cuda(), None, None, buf[:, :D], groups, eps, seq_ops.GATE_NONE)
    assert worst_row(buf[:, :D].float(), O.over_rms(o.view(rows, groups, size), eps).reshape(rows, D)) < (1e-5 if f32 else 1e-2)
    assert bool((buf[:, D:] == 3.0).all())


@pytest.mark.parametrize("H,G,dim,vdim,rot", [(4, 2, 24, 20, 12), (6, 3, 64, 64, 64), (3, 1, 9, 5, 4), (2, 2, 96, 64, 40), (1, 1, 2, 1, 2), (8, 2, 128, 128, 0)])
@pytest.mark.parametrize("f32", [True, False])
def test_attention_front_end(H, G, dim, vdim, rot, f32):
    """Norms over the whole projections, rotation with a gain at positions in the thousands, blended values, rows into the right pages."""
    from paligemma_multimodal_system_b200 import seq_ops
    dt, eps, lam, ctx, n = (F32 if f32 else BF16), 1e-2, 0.3, 5000, 70
    g = torch.Generator().manual_seed(H * dim)
    r = {"base": 300.0, "dims": rot, "scaling": {"factor": 4.0, "original": 200, "fast": 8.0, "slow": 1.0}}
    f, gain = O.frequencies(r) if rot else ([0.0], 1.0)
    W = (H + G) * dim + G * vdim
    x, other = torch.randn(n, W + 3, generator=g).to(BF16).float(), torch.randn(n, G * vdim + 2, generator=g).to(BF16).float()
    qn, kn = torch.randn(H * dim, generator=g), torch.randn(G * dim, generator=g)
    pages = [3, 0, 2]
    table = [1] * (ctx // 64) + pages
    kp, vp = (torch.full((4, 64, G * s), 7.0, device="cuda", dtype=dt) for s in (dim, vdim))
    b = seq_ops.make_step_batch([dict(tokens=[0] * n, ctx=ctx, slot=0, pages=table)])
    q_out = torch.empty(n, H * dim, device="cuda", dtype=dt)
    freq = torch.tensor(f, dtype=torch.float64).cuda()
    seq_ops.attn_prepare(x.cuda().to(dt), b, freq, qn.cuda(), kn.cuda(), q_out, kp, vp, H, G, dim, vdim, rot, eps, 64, norm_qk=seq_ops.NORM_PROJECTION, norm_v=False,
                         rot_gain=gain, v_other=other.cuda().to(dt)[:, 1:1 + G * vdim], v_mix=lam)
    xd = x.double()
    q = O.over_rms(xd[:, :H * dim], eps) * qn
    k = O.over_rms(xd[:, H * dim:(H + G) * dim], eps) * kn
    q = torch.stack([O.turned(q[t].view(H, dim), ctx + t, r, "next") for t in range(n)])
    k = torch.stack([O.turned(k[t].view(G, dim), ctx + t, r, "next") for t in range(n)])
    v = (1 - lam) * xd[:, (H + G) * dim:W] + lam * other.double()[:, 1:1 + G * vdim]
    rows = torch.tensor([table[(ctx + t) // 64] * 64 + (ctx + t) % 64 for t in range(n)])
    tol = 1e-5 if f32 else 1e-2
    assert worst_row(q_out.float(), q) < tol
    assert worst_row(kp.view(-1, G * dim)[rows.cuda()].float(), k) < tol and worst_row(vp.view(-1, G * vdim)[rows.cuda()].float(), v) < tol
    left = torch.ones(4 * 64, dtype=torch.bool)
    left[rows] = False
    assert bool((kp.view(4 * 64, -1)[left.cuda()] == 7.0).all()) and bool((vp.view(4 * 64, -1)[left.cuda()] == 7.0).all())


MIXERS = [attention(v_mix=False), attention(heads=6, kv_heads=1, dim=64, vdim=64, rot_dims=32, size=65, keep_first=0), attention(heads=2, kv_heads=2, dim=96, vdim=64, rot_dims=96, size=None, scaling=None),
          attention(heads=3, kv_heads=3, dim=7, vdim=5, rot_dims=2, size=1, keep_first=2, v_mix=False), attention(heads=4, kv_heads=2, dim=128, vdim=128, rot_dims=0, size=64, keep_first=64),
          attention(heads=1, kv_heads=1, dim=40, vdim=80, size=300, keep_first=1, scale=0.5), attention(heads=2, kv_heads=1, dim=32, vdim=32, rot_dims=32, size=20, keep_first=130),
          retention(), retention(heads=6, dim=64, vdim=32, rot_dims=64), retention(heads=2, dim=40, vdim=64, rot_dims=16), retention(heads=3, dim=5, vdim=11, rot_dims=2, decay=[1.0, 0.3, 0.999]),
          retention(heads=2, dim=128, vdim=136, rot_dims=0), retention(heads=1, dim=96, vdim=96, rot_dims=96, decay=[0.98])]


@pytest.mark.parametrize("mi", range(len(MIXERS)))
@pytest.mark.parametrize("dtype,tol", [(F32, 5e-5), (BF16, 4e-2)])
def test_mixer_alone_whole_in_portions_and_token_by_token(mi, dtype, tol):
    from paligemma_multimodal_system_b200 import seq_ops
    D, T, eps, l = 56, 150, 1e-4, MIXERS[mi]
    first = bare(dict(l)) if l["mixer"].get("v_mix") else None  # a blending layer reads an earlier one's values
    cfg = make_cfg(([first] if first else []) + [bare(l)], width=D, eps=eps)
    i = len(cfg["layers"]) - 1
    w = O.random_weights(cfg, seed=mi)
    g = torch.Generator().manual_seed(mi)
    h = torch.randn(T, D, generator=g).to(BF16).float()
    wd, hd = {k: v.double() for k, v in w.items()}, h.double()
    other = None
    if l["type"] == "attention":
        other = torch.randn(T, l["mixer"]["kv_heads"] * l["mixer"]["vdim"], generator=g).to(BF16).float() if first else None
        ref = O.attention(hd, wd, f"l{i}.mix.", l["mixer"], eps, None if other is None else other.double())[0]
    else:
        ref = O.retention(hd, wd, f"l{i}.mix.", l["mixer"], eps)
    mx = load_mixer(cfg, w, i)
    prec = seq_ops.Precision(dtype)
    mx.pack(prec)
    for cuts in ([T], [70, 16, 2, 1], [2], [15, 17], [149, 1]):
        got = run_mixer(mx, h, cuts, dtype, prec, other)
        assert median_row(got, ref) < tol / 2 and worst_row(got, ref) < 2 * tol, (cuts, median_row(got, ref), worst_row(got, ref))


@pytest.mark.parametrize("size,keep", [(1, 0), (31, 3), (64, 0), (65, 70), (100, 1), (128, 64)])
@pytest.mark.parametrize("dtype,dim,vdim", [(F32, 20, 12), (BF16, 64, 64), (BF16, 20, 12), (BF16, 96, 64)])
def test_window_edges_and_kept_tokens_with_one_key_that_stands_out(size, keep, dtype, dim, vdim):
    """Every query looks along one direction and one token's key lies on it, with a large value: the row shows at once whether that token was
    visible.  Marked tokens at page and tile borders, among the kept first ones and just behind them; queries one inside and one outside the
    window (every row is compared); read by prompt rows, by portions and by decoded tokens."""
    from paligemma_multimodal_system_b200 import seq_ops
    H, G, D, T, eps = 2, 1, 48, 210, 1e-5
    l = attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, size=size, keep_first=keep, rot_dims=4, v_mix=False, scale=40.0 / dim)
    cfg = make_cfg([bare(l)], width=D, eps=eps)
    prec = seq_ops.Precision(dtype)
    for mark in sorted({0, max(keep - 1, 0), keep, keep + 1, 31, 32, 63, 64, 100}):
        w = O.random_weights(cfg, seed=mark)
        g = torch.Generator().manual_seed(mark)
        along = torch.zeros(dim)
        along[4:] = torch.sign(torch.randn(dim - 4, generator=g))  # the turned dimensions stay out of it
        # column 0 of h is one everywhere and makes the query, column 1 marks the token, the others are noise
        wq, wk, wv = 0.05 * w["l0.mix.q"], w["l0.mix.k"].clone(), w["l0.mix.v"].clone()
        wq[:, 0], wk[:, 0], wk[:, 1] = along.repeat(H), 0.0, 30.0 * along
        wv[:, 0], wv[:, 1] = 0.0, 6.0
        w.update({"l0.mix.q": wq.to(BF16).float(), "l0.mix.k": wk.to(BF16).float(), "l0.mix.v": wv.to(BF16).float(),
                  "l0.mix.q.norm": torch.ones(H * dim), "l0.mix.k.norm": torch.ones(G * dim)})
        h = 0.3 * torch.randn(T, D, generator=g)
        h[:, 0], h[:, 1] = 1.0, 0.0
        h[mark, 1] = 1.0
        h = h.to(BF16).float()
        ref = O.attention(h.double(), {k: v.double() for k, v in w.items()}, "l0.mix.", l["mixer"], eps)[0]
        size_of = ref.pow(2).mean(-1).sqrt()
        seen = torch.tensor([O.visible(i, mark, l["mixer"]["mask"]) for i in range(T)])
        if size > 1 and bool((~seen[mark:]).any()):
            assert float(size_of[seen].min()) > 1.5 * float(size_of[~seen].max())  # the data do tell
        mx = load_mixer(cfg, w)
        mx.pack(prec)
        for cuts in ([T], [90, 2, 1], [mark + size, 1, 40] if mark + size < T else [64, 65]):
            assert worst_row(run_mixer(mx, h, cuts, dtype, prec), ref) < (1e-4 if dtype == F32 else 3e-2), (mark, cuts)


@pytest.mark.parametrize("experts,top,groups", [(8, 3, (4, 2)), (16, 4, (2, 1)), (9, 1, (3, 1)), (5, 5, None), (64, 8, (8, 3)), (130, 40, (2, 2)), (6, 2, (6, 3)), (1, 1, None)])
def test_router_choice_weights_and_counts(experts, top, groups):
    """Logistic scores, groups ranked by their two best, weights as they are: against the oracle token by token; half of the tokens have a group
    whose single best expert is the best of all while another group holds the best pair."""
    from paligemma_multimodal_system_b200 import seq_ops
    T = 60
    g = torch.Generator().manual_seed(experts)
    z = torch.randn(T, experts, generator=g)
    if groups and experts // groups[0] > 1:
        size = experts // groups[0]
        z[::2] -= 2.0
        z[::2, 0], z[::2, size:size + 2] = 3.0, torch.tensor([1.5, 1.6])
    count, keep = groups or (1, 1)
    pad = torch.full((T, experts + 3), 50.0)
    pad[:, :experts] = z
    flags = seq_ops.ROUTE_LOGISTIC | seq_ops.ROUTE_GROUP_BEST_TWO | seq_ops.ROUTE_PLAIN_WEIGHTS
    ids, wts, counts = seq_ops.moe_route(pad.cuda()[:, :experts], None, experts, top, count, keep, 1.0, flags=flags)
    router = {"experts": experts, "top": top, **({"groups": {"count": count, "keep": keep}} if groups else {})}
    n = [0] * experts
    for t in range(T):
        want = O.chosen(z[t], router)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(wts[t].cpu(), torch.stack([s for _, s in want]), atol=1e-6)
        for e, _ in want:
            n[e] += 1
    assert counts.tolist() == n


def load_ff(cfg, w, prec):
    from paligemma_multimodal_system_b200.modeling_padulorn import _feed_forward
    ff = _feed_forward(cfg["width"], cfg["layers"][0]["mlp"])
    left = {k: v.to(BF16) for k, v in w.items()}
    ff.load(lambda name, shape: left.pop(name), "l0.mlp.")
    ff.pack(prec)
    return ff


@pytest.mark.parametrize("width,kw", [(64, dict()), (50, dict(experts=6, top=2, ff=33, groups=None)), (128, dict(experts=4, top=2, ff=128, groups=(2, 1))), (24, dict(experts=3, top=3, ff=1, groups=None)),
                                      (72, dict(experts=70, top=6, ff=16, groups=(7, 3)))])
@pytest.mark.parametrize("dtype,T", [(F32, 77), (BF16, 77), (F32, 1), (BF16, 1), (BF16, 700)])
def test_experts_alone_and_with_the_norm_and_residual(width, kw, dtype, T):
    """(700 tokens over few experts: the gathered per-expert dense products.)"""
    from paligemma_multimodal_system_b200 import seq_ops
    cfg = make_cfg([moe(retention(), **kw)], width=width)
    w = O.random_weights(cfg, seed=T)
    g = torch.Generator().manual_seed(5)
    h, x0, nw = torch.randn(T, width, generator=g).to(BF16).float(), torch.randn(T, width, generator=g), torch.randn(width, generator=g)
    prec = seq_ops.Precision(dtype)
    ff = load_ff(cfg, w, prec)
    hd = h.cuda().to(dtype).contiguous()
    ref = O.experts(h.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", cfg["layers"][0]["mlp"])
    tol = 1e-5 if dtype == F32 else 1.5e-2
    assert worst_row(ff(hd, None, prec), ref) < tol
    eps = 1e-2
    want = x0 + O.over_rms(ref, eps) * nw
    for out in (torch.empty(T, width, device="cuda", dtype=dtype), None):
        x = x0.cuda().contiguous()
        ff.add_normed(hd, prec, nw.cuda(), x, out, eps)
        assert worst_row(x, want) < tol and (out is None or worst_row(out.float(), want) < tol)


def test_gelu_is_the_erf_form():
    """Where the two forms differ most (3e-4 near 2.2) fp32 experts must follow erf."""
    from paligemma_multimodal_system_b200 import seq_ops
    cfg = make_cfg([moe(retention(), 1, 1, 8, None)], width=8)
    w = {k: torch.zeros_like(v) for k, v in O.random_weights(cfg).items()}
    w["l0.mlp.e0.up"], w["l0.mlp.e0.down"] = torch.eye(8), torch.eye(8)
    h = torch.linspace(-4, 4, 8 * 50).view(50, 8)
    prec = seq_ops.Precision(F32)
    got = load_ff(cfg, w, prec)(h.cuda(), None, prec).cpu()
    assert float((got - 0.5 * O.gelu_erf(h.double())).abs().max()) < 1e-6  # the zero router weighs with sigmoid(0)


@pytest.mark.parametrize("rows,D,col0,scale", [(5, 72, 0, 3.7), (1, 33, 0, 1.0), (40, 64, 16, 0.25)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_rows_and_their_copy(rows, D, col0, scale, dtype):
    from paligemma_multimodal_system_b200 import seq_ops
    g = torch.Generator().manual_seed(D)
    table = torch.randn(50, D + col0, generator=g).to(BF16)
    tk = torch.randint(0, 50, (rows,), generator=g)
    copy = torch.empty(rows, D, device="cuda", dtype=dtype)
    x = seq_ops.embed_rows(tk.int().cuda(), table.cuda().to(dtype), col0, D, scale, out_act=copy)
    want = table.float()[tk][:, col0:] * scale
    assert torch.equal(x.cpu(), want) and torch.equal(copy.cpu(), want.to(dtype))


# ----------------------------------------------------------------------------------------------------------------------
# whole models
# ----------------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def base():
    w = steady_weights(BASE_CFG, seed=2)
    tk = toks(150, BASE_CFG["vocab"], 2)
    return w, tk, O.forward(BASE_CFG, w, tk)


def test_routers_that_read_the_whole_residual():
    """Unconstrained random routers (close calls included) in fp32, layer by layer."""
    w, tk = O.random_weights(BASE_CFG, seed=3), toks(120, BASE_CFG["vocab"], 4)
    eng = engine_for(BASE_CFG, w, F32)
    poison(eng)
    trace = []
    got = eng.step([("a", tk, list(range(len(tk))))], ["a"], trace=trace)
    ref, layers = O.forward(BASE_CFG, w, tk, return_layers=True)
    assert all(close(x, y, F32) for x, y in zip(trace, layers)) and close(got, ref, F32)
    eng = engine_for(BASE_CFG, w, F32)
    poison(eng)
    assert close(run_cut(eng, "a", tk, [50, 3, 1, 40]), ref, F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_whole_prompt_every_layer(base, dtype):
    w, tk, ref = base
    eng = engine_for(BASE_CFG, w, dtype)
    poison(eng)
    trace = []
    got = eng.step([("a", tk, list(range(len(tk))))], ["a"], trace=trace)
    _, layers = O.forward(BASE_CFG, w, tk, return_layers=True)
    assert len(trace) == len(BASE_CFG["layers"])
    for i, x in enumerate(trace):
        assert close(x, layers[i], dtype), f"residual after layer {i}"
    assert close(got, ref, dtype)


@pytest.mark.parametrize("cuts", [[1], [2], [3, 5, 2], [31, 33], [32], [64, 1], [65, 2, 2, 1], [100, 7], [15, 16, 17]])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_portions_and_token_by_token_equal_the_whole_prompt(base, cuts, dtype):
    w, tk, ref = base
    eng = engine_for(BASE_CFG, w, dtype)
    poison(eng)
    assert close(run_cut(eng, "a", tk, cuts), ref, dtype)


def test_causal_edge_and_stale_rows(base):
    """Position i must see row i and not row i + 1: a changed LAST token leaves every earlier position's logits bit-identical."""
    w, _, _ = base
    tk = toks(80, BASE_CFG["vocab"], 6)
    eng = engine_for(BASE_CFG, w, F32)
    poison(eng)
    got = eng.step([("a", tk, list(range(80)))], ["a"])
    tk2 = tk[:-1] + [(tk[-1] + 1) % BASE_CFG["vocab"]]
    got2 = eng.step([("b", tk2, list(range(80)))], ["b"])
    assert torch.equal(got[:-1], got2[:-1]) and not torch.equal(got[-1], got2[-1])
    assert close(got, O.forward(BASE_CFG, w, tk), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_batch_equals_each_alone_and_pages_and_slots_are_reused(base, dtype):
    """Four live requests of different lengths, portions beside single tokens, in a pool that only holds them because finished
    requests give their pages and slots back; every request's logits equal its solo run."""
    w, _, _ = base
    V = BASE_CFG["vocab"]
    prompts = {i: toks(n, V, 10 + i) for i, n in enumerate([130, 70, 1, 45, 90, 64, 3])}
    refs = {i: O.forward(BASE_CFG, w, p) for i, p in prompts.items()}
    eng = engine_for(BASE_CFG, w, dtype, max_tokens=6 * 64, slots=4)
    poison(eng)
    fed = {i: 0 for i in prompts}
    got = {i: [] for i in prompts}
    waiting, live, step = list(prompts), [], 0
    seen_pages, seen_slots = {}, {}
    while waiting or live:
        while waiting and len(live) < 4 and sum((len(prompts[i]) + 63) // 64 for i in live + waiting[:1]) <= 6:
            live.append(waiting.pop(0))
        entries, end = [], []
        for k, i in enumerate(live):
            if (step + 2 * k) % 7 == 6 and len(live) > 1:
                continue  # sits this step out: its state must be there again afterwards
            left = len(prompts[i]) - fed[i]
            n = 1 if (step + k) % 3 == 0 else min(left, [17, 2, 40][(step + k) % 3])
            n = min(n, left)
            entries.append((i, prompts[i][fed[i]:fed[i] + n], list(range(n))))
            fed[i] += n
            if fed[i] == len(prompts[i]):
                end.append(i)
        out = eng.step(entries, end)
        for i in live:
            if i in eng.store.live:
                seen_pages[i], seen_slots[i] = list(eng.store.live[i].pages), eng.store.live[i].slot
        r = 0
        for i, tk, _ in entries:
            got[i].append(out[r:r + len(tk)])
            r += len(tk)
        live = [i for i in live if i not in end]
        step += 1
    for i in prompts:
        assert close(torch.cat(got[i]), refs[i], dtype), i
    all_pages = [p for ps in seen_pages.values() for p in ps]
    assert len(all_pages) > len(set(all_pages)), "no page was handed out twice"
    assert len(set(seen_slots.values())) < len(seen_slots), "no slot was handed out twice"
    assert not eng.store.live and len(eng.store.pool.free) == 6


def test_long_decoding_across_page_borders_and_out_of_the_window(base):
    w, _, _ = base
    tk = toks(260, BASE_CFG["vocab"], 77)
    ref = O.forward(BASE_CFG, w, tk)
    for dtype in (F32, BF16):
        eng = engine_for(BASE_CFG, w, dtype)
        poison(eng)
        assert close(run_cut(eng, "a", tk, [60, 1]), ref, dtype)  # 200 single-token steps: eager, captured, then replayed graphs


def test_decoded_batches_of_one_geometry_share_a_graph_but_not_their_values(base):
    """A replayed decode graph serves other requests than the ones it was captured with: rotation tables and the blended layer's values belong
    to the step, not to the capture."""
    w, _, _ = base
    V = BASE_CFG["vocab"]
    eng = engine_for(BASE_CFG, w, F32, slots=2)
    poison(eng)
    for pair in range(3):
        ps = [toks(30 + 7 * pair, V, 60 + pair), toks(45 - 9 * pair, V, 70 + pair)]
        refs = [O.forward(BASE_CFG, w, p) for p in ps]
        eng.step([(i, p[:-6], []) for i, p in enumerate(ps)])
        for t in range(6):
            out = eng.step([(i, [p[len(p) - 6 + t]], [0]) for i, p in enumerate(ps)], [0, 1] if t == 5 else [])
            assert close(out, torch.stack([refs[i][len(p) - 6 + t] for i, p in enumerate(ps)]), F32), (pair, t)


def test_first_tokens_of_a_sequence(base):
    """One-token prompts, a one-token first portion, two-token portions from the start."""
    w, tk, ref = base
    eng = engine_for(BASE_CFG, w, F32)
    poison(eng)
    one = eng.step([("x", tk[:1], [0])], ["x"])
    assert close(one, ref[:1], F32)
    assert close(run_cut(eng, "y", tk[:9], [1, 2, 2, 1, 3]), ref[:9], F32)
    assert close(run_cut(eng, "z", tk[:8], [2]), ref[:8], F32)


OTHER_SIZES = [
    # odd sizes the 16-byte paths cannot take
    make_cfg([moe(attention(heads=3, kv_heads=3, dim=10, vdim=7, rot_dims=6, size=11, keep_first=2), 5, 2, 25, None), bare(retention(heads=3, dim=10, vdim=7, rot_dims=6)),
              moe(attention(heads=3, kv_heads=1, dim=14, vdim=21, rot_dims=2, size=40, keep_first=0), 6, 2, 11, (2, 1))], width=34, vocab=41, embed=1.0, mult=1.0, logit=1.0),
    # sizes the tensor-core kernels like
    make_cfg([moe(retention(heads=4, dim=128, vdim=64, rot_dims=128), 8, 2, 64, (2, 1)), moe(attention(heads=4, kv_heads=1, dim=128, vdim=128, rot_dims=64, size=50, keep_first=4), 8, 2, 128, None),
              moe(attention(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=64, size=None), 16, 4, 32, (8, 4))], width=128, vocab=256, eps=1e-6, mult=0.4),
    # a single head everywhere, no rotation, no window, one expert, constants of one; retention only at the end
    make_cfg([bare(attention(heads=1, kv_heads=1, dim=2, vdim=1, rot_dims=0, size=None, v_mix=False)), moe(retention(heads=1, dim=2, vdim=4, rot_dims=2, decay=[1.0]), 1, 1, 12, None),
              bare(retention(heads=1, dim=1, vdim=3, rot_dims=0, decay=[0.2]))], width=24, vocab=20, embed=1.0, mult=1.0, logit=1.0),
    # every layer blends; windows shorter than what is kept; a window of one
    make_cfg([moe(attention(size=3, keep_first=20), 4, 2, 16, (2, 1)), moe(attention(size=1, keep_first=0), 4, 4, 16, None), bare(attention(heads=8, kv_heads=4, vdim=10, size=90, keep_first=64)),
              moe(attention(size=16, keep_first=16), 10, 3, 8, (5, 2))], mult=1.3, logit=3.0),
]


@pytest.mark.parametrize("ci", range(len(OTHER_SIZES)))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_other_sizes(ci, dtype):
    cfg = OTHER_SIZES[ci]
    w = steady_weights(cfg, seed=20 + ci)
    tk = toks(130, cfg["vocab"], ci)
    ref = O.forward(cfg, w, tk)
    eng = engine_for(cfg, w, dtype)
    poison(eng)
    got = run_cut(eng, "a", tk, [70, 2, 1, 1, 20, 1])
    if ci == 2 and dtype == BF16:  # heads of one or two elements: norms of nearly vanishing vectors amplify the rounding of single rows
        assert median_row(got, ref) < BF16_TOL
        return
    assert close(got, ref, dtype)
    two = [toks(n, cfg["vocab"], 50 + n) for n in (66, 30)]
    out = eng.step([(i, p, list(range(len(p)))) for i, p in enumerate(two)], [0, 1])
    assert close(out[:66], O.forward(cfg, w, two[0]), dtype) and close(out[66:], O.forward(cfg, w, two[1]), dtype)


GEN_CFG = make_cfg([moe(attention(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=8, size=30, keep_first=2), 4, 2, 24, (2, 1)), moe(retention(heads=2, dim=16, vdim=16), 4, 1, 32, None),
                    bare(attention(heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=8, size=12, keep_first=1))], width=48, vocab=60)


def greedy(cfg, w, prompt, new, margin=1e-3):
    seq = list(prompt)
    for _ in range(new):
        lg = O.forward(cfg, w, seq)[-1]
        top2 = lg.topk(2).values
        assert float(top2[0] - top2[1]) > margin, "test weights give a near tie"
        seq.append(int(lg.argmax()))
    return seq[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """engine.generate: more prompts than slots, a pool smaller than the sum of all requests, portions of 48 rows; the tokens
    equal the oracle's greedy continuation of each prompt alone."""
    w = O.random_weights(GEN_CFG, seed=31)
    prompts = [toks(n, 60, 40 + n) for n in (70, 5, 33, 1, 90, 12)]
    eng = engine_for(GEN_CFG, w, F32, max_tokens=5 * 64, slots=3)
    poison(eng)
    got = eng.generate(prompts, 10, step_tokens=48)
    for p, g in zip(prompts, got):
        assert g == greedy(GEN_CFG, w, p, 10)
    assert not eng.store.live and len(eng.store.pool.free) == 5


def test_sampled_generation_stays_in_vocabulary_and_stops_at_eos():
    w = O.random_weights(GEN_CFG, seed=9)
    eng = engine_for(GEN_CFG, w, BF16, max_tokens=256, slots=2)
    out = eng.generate([toks(20, 60, 1), toks(3, 60, 2), toks(40, 60, 3)], 10, do_sample=True, temperature=0.9, top_p=0.8, eos_token_id=7, seed=3)
    for g in out:
        assert 1 <= len(g) <= 10 and all(0 <= t < 60 for t in g)
        assert 7 not in g[:-1]


def write_checkpoint(path, cfg, w):
    meta, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(BF16).contiguous().view(torch.int16).numpy().tobytes()
        meta[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(meta).encode()
    path.mkdir(exist_ok=True)
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    (path / "config.json").write_text(json.dumps(cfg))


def test_registry_and_command_line_serve_a_checkpoint_folder(tmp_path):
    """config.json + model.safetensors on disk -> registry.load_model -> the same logits as the oracle; inference.main generates from it."""
    from paligemma_multimodal_system_b200 import inference
    from paligemma_multimodal_system_b200.engine import SequenceEngine
    from paligemma_multimodal_system_b200.registry import load_model
    w = O.random_weights(GEN_CFG, seed=31)
    write_checkpoint(tmp_path / "m", GEN_CFG, w)
    tk = toks(50, 60, 5)
    eng = SequenceEngine(load_model(str(tmp_path / "m"), dtype=F32), 128, 1)
    assert close(eng.step([("a", tk, list(range(50)))], ["a"]), O.forward(GEN_CFG, w, tk), F32)
    prompts = [toks(5, 60, 45), toks(33, 60, 73)]
    got = inference.main(str(tmp_path / "m"), prompt_ids=";".join(" ".join(map(str, p)) for p in prompts), max_tokens_to_generate=4, dtype="float32")
    for p, g in zip(prompts, got):
        assert g == greedy(GEN_CFG, w, p, 4)


def test_wider_model_long_prompt_reaches_the_large_tile_paths():
    """Width 512, tensor-core head sizes and per-expert dense products over 1100 tokens in bf16; then 20 decoded tokens beyond the window."""
    cfg = make_cfg([moe(retention(heads=8, dim=64, vdim=64, rot_dims=64), 4, 2, 256, (2, 1)), moe(attention(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=32, size=300, keep_first=8), 8, 2, 512, (4, 2)),
                    bare(attention(heads=6, kv_heads=2, dim=96, vdim=64, rot_dims=48, size=None))], width=512, vocab=1000)
    w = steady_weights(cfg, seed=77)
    tk = toks(1120, 1000, 3)
    ref = O.forward(cfg, w, tk, dtype=F32)
    eng = engine_for(cfg, w, BF16, max_tokens=1280, slots=2)
    poison(eng)
    assert close(run_cut(eng, "a", tk, [1100, 1]), ref, BF16)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_a_mixed_schedule(tmp_path, dtype):
    """bin/trace_run on a checkpoint folder: portions beside single tokens, a step that wants nothing, a request that sits out a step,
    a finished request's page and slot taken over by a later one; the written logits equal the oracle's for each request alone."""
    import subprocess
    import numpy as np
    cfg = OTHER_SIZES[0]
    w = steady_weights(cfg, seed=13)
    write_checkpoint(tmp_path / "model", cfg, w)
    V = cfg["vocab"]
    tk = {"a": toks(70, V, 1), "b": toks(33, V, 2), "c": toks(1, V, 3), "d": toks(20, V, 4)}
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": tk["a"][:40], "want": [0, 39]}, {"id": "b", "tokens": tk["b"][:2], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": tk["a"][40:41], "want": [0]}, {"id": "c", "tokens": tk["c"], "want": [0]}], "end": ["c"]},
        {"step": 2, "entries": [{"id": "b", "tokens": tk["b"][2:32], "want": []}, {"id": "a", "tokens": tk["a"][41:42], "want": []}], "end": []},
        {"step": 3, "entries": [{"id": "d", "tokens": tk["d"][:19], "want": [18]}, {"id": "a", "tokens": tk["a"][42:], "want": [27]}, {"id": "b", "tokens": tk["b"][32:], "want": [0]}],
         "end": ["a", "b"]},
        {"step": 4, "entries": [{"id": "d", "tokens": tk["d"][19:], "want": [0]}], "end": ["d"]},
    ]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(5)]
    assert not (out / "2.f32").exists()
    ref = {k: O.forward(cfg, w, v) for k, v in tk.items()}
    want = {0: [("a", 0), ("a", 39), ("b", 1)], 1: [("a", 40), ("c", 0)], 3: [("d", 18), ("a", 69), ("b", 32)], 4: [("d", 19)]}
    dt = F32 if dtype == "float32" else BF16
    for step, rows in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        assert close(got, torch.stack([ref[k][p] for k, p in rows]), dt), step
