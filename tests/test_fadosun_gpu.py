"""Fadosun through the framework (kernels, page pool and state slots, ragged steps, scheduler) against the plain oracle
(oracle/fadosun_oracle.py): every mechanism alone, then whole models under every way of cutting and batching the work."""
import json
import os
import struct
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from oracle import fadosun_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 2e-4, 4e-2


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=4):
    return {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def parallel(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=8, base=400.0, scale=None, rheads=6, groups=3, state=20, rvdim=12, conv=4, norm_groups=4, ls=1.3, rs=0.6):
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot={"base": base, "dims": rot_dims}, scale=scale if scale is not None else dim ** -0.5)
    right = dict(heads=rheads, groups=groups, state=state, vdim=rvdim, conv=conv, norm_groups=norm_groups)
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs}}


def memory(heads=3, dim=20, vdim=28, cap=9.0):
    return {"type": "mlstm", "mixer": dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)}


def with_ff(l, ff=80):
    return dict(l, mlp={"kind": "dense", "ff": ff} if ff else None)


def make_cfg(layers, width=72, vocab=90, eps=1e-5):
    return {"architecture": "Fadosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every mixer type, shared and own query/key heads, a layer without a feed-forward
BASE_CFG = make_cfg([with_ff(delta()), with_ff(parallel()), with_ff(memory(), 0), with_ff(delta(heads=3, kv_heads=3, dim=16, vdim=32, conv=3), 48),
                     with_ff(parallel(heads=3, kv_heads=3, dim=20, vdim=12, rot_dims=20, rheads=4, groups=1, state=9, rvdim=18, norm_groups=1), 33)])


def build(cfg, w, dtype):
    from paligemma_multimodal_system_b200.modeling_fadosun import FadosunConfig, FadosunForCausalLM
    return FadosunForCausalLM(FadosunConfig(cfg), dtype).load_weights({k: v.to(torch.bfloat16) for k, v in w.items()})


def engine_for(cfg, w, dtype, max_tokens=1024, slots=4):
    from paligemma_multimodal_system_b200.engine import SequenceEngine
    return SequenceEngine(build(cfg, w, dtype), max_tokens, slots)


def poison(engine):
    """Stale memory must never be read: pages and state slots start as huge values instead of zeros."""
    for t in engine.store.k_pages + engine.store.v_pages + engine.store.state:
        if t is not None:
            t.fill_(1e4)


def rel_err(got, ref):
    got, ref = got.double().cpu(), ref.double()
    return float((got - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt())


def worst_row(got, ref):
    """The largest error of any row, relative to the typical row's size (one wrong position must not drown among hundreds)."""
    got, ref = got.double().cpu().reshape(ref.shape[0], -1), ref.double().reshape(ref.shape[0], -1)
    return float(((got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()).max())


def close(got, ref, dtype):
    """fp32: every row within F32_TOL.  bf16: the tensor within BF16_TOL and no row beyond twice that."""
    if dtype == torch.float32:
        return worst_row(got, ref) < F32_TOL
    return rel_err(got, ref) < BF16_TOL and worst_row(got, ref) < 2 * BF16_TOL


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


def run_mixer(mx, h, cuts, dtype, prec):
    """h [T, D] through a mixer in portions; returns fp32 [T, D] on the CPU."""
    from paligemma_multimodal_system_b200 import seq_ops
    T = h.shape[0]
    store = one_store(mx.cache_specs(), T, dtype)
    rec, pos, outs, i = store.live[0], 0, [], 0
    while pos < T:
        k = min(cuts[min(i, len(cuts) - 1)], T - pos)
        b = seq_ops.make_step_batch([dict(tokens=[0] * k, ctx=pos, slot=rec.slot, pages=rec.pages)])
        outs.append(mx(h[pos:pos + k].cuda().to(dtype).contiguous(), b, store, 0, prec).float().cpu())
        pos, i = pos + k, i + 1
    return torch.cat(outs)


def load_mixer(cfg, w, i=0):
    from paligemma_multimodal_system_b200.modeling_fadosun import _mixer
    l = cfg["layers"][i]
    mx = _mixer(cfg["width"], l["type"], l["mixer"], cfg["norm"]["eps"])
    left = {k: v.to(torch.bfloat16) for k, v in w.items()}
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
LENS, PLANS = [83, 9, 46], [[5, 1, 2, 75], [1] * 9, [2, 2, 1, 3, 38]]


@pytest.mark.parametrize("sizes,taps", [(((3, 16), (3, 16), (5, 24)), 4), (((2, 7), (2, 7), (1, 9)), 3), (((1, 130), (1, 130), (4, 64)), 8), (((2, 64), (2, 64), (2, 64)), 1),
                                        (((1, 300), (1, 300), (1, 50)), 2)])
@pytest.mark.parametrize("f32", [True, False])
def test_short_convolution_in_portions(sizes, taps, f32):
    """Three sequences advance together in unequal portions (one token by token, one in portions shorter than the convolution's reach): the
    activations and the inverse norms of the first two sections must equal the whole-sequence oracle, whatever the slots held before."""
    from paligemma_multimodal_system_b200 import seq_ops
    dt = torch.float32 if f32 else torch.bfloat16
    g = torch.Generator().manual_seed(taps + sizes[0][1])
    counts = [n * s for n, s in sizes]
    at = [0, (counts[0] + 7) // 8 * 8]
    at.append(at[1] + (counts[1] + 7) // 8 * 8)
    C = at[2] + (counts[2] + 7) // 8 * 8
    xs = [torch.randn(n, C, generator=g).to(torch.bfloat16).float() for n in LENS]
    w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    ref = [O.silu(O.short_conv(x, w, bias)) for x in xs]
    sec = seq_ops.ConvSections([dict(groups=n, size=s, xcol=a + 8, ccol=a, unit=i < 2, scale=0.5 if i == 0 else 1.0) for i, ((n, s), a) in enumerate(zip(sizes, at))])
    state = torch.full((4, taps - 1, C), 1e4, device="cuda") if taps > 1 else None
    wd, bd = w.t().contiguous().cuda(), bias.cuda()
    got, inv = [[] for _ in LENS], [[] for _ in LENS]
    for rows, b in ragged(LENS, PLANS):
        x = torch.zeros(b.T, C + 16)
        x[:, 8:C + 8] = torch.cat([xs[i][p:p + k] for i, p, k in rows])
        out, iv = torch.empty(b.T, C, device="cuda", dtype=dt), torch.empty(b.T, sizes[0][0] + sizes[1][0], device="cuda")
        seq_ops.short_conv(x.cuda().to(dt), wd, state, out, sec, b, bias=bd, inv=iv)
        r = 0
        for i, _, k in rows:
            got[i].append(out[r:r + k].float().cpu())
            inv[i].append(iv[r:r + k].cpu())
            r += k
    for i in range(3):
        y, v = torch.cat(got[i]), torch.cat(inv[i])
        for a, c in zip(at, counts):
            assert worst_row(y[:, a:a + c], ref[i][:, a:a + c]) < (1e-5 if f32 else 1e-2), i
        for s in range(2):
            n, size = sizes[s]
            want = (0.5 if s == 0 else 1.0) / torch.sqrt((ref[i][:, at[s]:at[s] + counts[s]].reshape(-1, n, size) ** 2).sum(-1) + 1e-6)
            have = v[:, s * sizes[0][0]:s * sizes[0][0] + n]
            assert float(((have - want) / want).abs().max()) < (1e-5 if f32 else 2e-2)


HEADS = [(4, 2, 24, 20), (3, 1, 64, 64), (2, 2, 48, 128), (2, 1, 128, 72), (5, 5, 7, 9), (1, 1, 100, 33), (2, 2, 200, 16)]
BLOCK_PLANS = [[83], [9], [16, 17, 13]]


@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
@pytest.mark.parametrize("f32,plans", [(True, PLANS), (False, PLANS), (False, BLOCK_PLANS)])
@pytest.mark.parametrize("strength", [0.5, 6.0])
def test_delta_rule(H, G, dim, vdim, f32, plans, strength):
    """Scan and block kernels (the latter with entries shorter, equal to and longer than a block) against the recurrence; decays from
    near one down to e^-40 per token."""
    from paligemma_multimodal_system_b200 import seq_ops
    dt = torch.float32 if f32 else torch.bfloat16
    g = torch.Generator().manual_seed(dim * vdim)
    rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    A, c = torch.rand(H, generator=g) - 1.0, torch.randn(H * dim, generator=g)
    Cq, Cv, Wb = (G * dim + 7) // 8 * 8, (H * vdim + 7) // 8 * 8, (H + 7) // 8 * 8
    data = [dict(q=rnd(n, Cq), k=rnd(n, Cq), v=rnd(n, Cv), b=rnd(n, Wb), a=strength * torch.randn(n, H * dim, generator=g)) for n in LENS]
    pick = torch.arange(H) // (H // G)
    ref, inv = [], []
    for d in data:
        n = d["q"].shape[0]
        q, k = (d[x][:, :G * dim].reshape(n, G, dim).double() for x in "qk")
        iq, ik = dim ** -0.5 / torch.sqrt((q * q).sum(-1) + 1e-6), 1.0 / torch.sqrt((k * k).sum(-1) + 1e-6)
        inv.append(torch.cat([iq, ik], 1).float())
        gd = torch.exp(-torch.exp(A.double())[:, None] * O.softplus(d["a"].double() + c.double()).view(n, H, dim))
        ref.append(O.delta_rule((q * iq[..., None])[:, pick], (k * ik[..., None])[:, pick], d["v"][:, :H * vdim].reshape(n, H, vdim).double(),
                                torch.sigmoid(d["b"][:, :H].double()), gd).reshape(n, H * vdim))
    state = torch.full((4, H, dim, vdim), 1e4, device="cuda")
    got = [[] for _ in LENS]
    for rows, b in ragged(LENS, plans):
        x = {key: torch.cat([data[i][key][p:p + k] for i, p, k in rows]).cuda() for key in "qkvba"}
        iv = torch.cat([inv[i][p:p + k] for i, p, k in rows]).cuda()
        out = torch.empty(b.T, H * vdim, device="cuda")
        seq_ops.delta_rule(x["q"].to(dt), x["k"].to(dt), x["v"].to(dt), x["b"].to(dt)[:, :H], iv, x["a"].contiguous(), A.cuda(), c.cuda(), state, out, b, H, G, dim, vdim)
        r = 0
        for i, _, k in rows:
            got[i].append(out[r:r + k].cpu())
            r += k
    for i in range(3):
        assert worst_row(torch.cat(got[i]), ref[i]) < 1e-4, i


@pytest.mark.parametrize("H,G,dim,vdim", HEADS)
@pytest.mark.parametrize("f32,plans", [(True, PLANS), (False, PLANS), (False, BLOCK_PLANS)])
@pytest.mark.parametrize("strength", [0.5, 6.0])
def test_state_space_and_matrix_memory_recurrences(H, G, dim, vdim, f32, plans, strength):
    from paligemma_multimodal_system_b200 import seq_ops
    dt_ = torch.float32 if f32 else torch.bfloat16
    g = torch.Generator().manual_seed(dim + vdim)
    rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    p1, p2, p3, cap = torch.randn(H, generator=g), torch.rand(H, generator=g) - 1.0, torch.randn(H, generator=g), 7.0
    Cq, Cv, Wb = (G * dim + 7) // 8 * 8, (H * vdim + 7) // 8 * 8, (H + 7) // 8 * 8
    data = [dict(q=rnd(n, Cq), k=rnd(n, Cq), v=rnd(n, Cv), i=(strength * rnd(n, Wb)).to(torch.bfloat16).float(), f=(strength * rnd(n, Wb)).to(torch.bfloat16).float())
            for n in LENS]
    pick = torch.arange(H) // (H // G)
    vb = seq_ops.recurrence_block(vdim)
    for kind in (seq_ops.STATE_SPACE, seq_ops.MATRIX_MEMORY):
        qs = 1.0 if kind == seq_ops.STATE_SPACE else dim ** -0.5
        ref, den = [], []
        for d in data:
            n = d["q"].shape[0]
            q, k = (d[x][:, :G * dim].reshape(n, G, dim).double()[:, pick] for x in "qk")
            v, gi, gf = d["v"][:, :H * vdim].reshape(n, H, vdim).double(), d["i"][:, :H].double(), d["f"][:, :H].double()
            if kind == seq_ops.STATE_SPACE:
                y = O.state_space(v, k, q, O.softplus(gi + p1.double()), torch.exp(p2.double())) + p3.double()[:, None] * v
            else:
                y = O.matrix_memory(q * qs, k, v, cap * torch.tanh((gi + p1.double()) / cap), -O.softplus(-cap * torch.tanh((gf + p2.double()) / cap)))
            ref.append(y)
        state = torch.full((4, H, dim, vdim), 1e4, device="cuda")
        norm = torch.full((4, -(-vdim // vb), H, dim + 1), 1e4, device="cuda")
        got = [[] for _ in LENS]
        for rows, b in ragged(LENS, plans):
            x = {key: torch.cat([data[i][key][p:p + k] for i, p, k in rows]).cuda().to(dt_) for key in "qkvif"}
            out = torch.empty(b.T, H * vdim, device="cuda")
            seq_ops.gated_recurrence(kind, x["q"], x["k"], x["v"], x["i"][:, :H], x["f"][:, :H], p1.cuda(), p2.cuda(), p3.cuda(), state, norm, out, b, H, G, dim, vdim,
                                     qscale=qs, cap=cap)
            r = 0
            for i, _, k in rows:
                got[i].append(out[r:r + k].cpu())
                r += k
        for i in range(3):
            y = torch.cat(got[i]).view(-1, H, vdim).double()
            # per token and head, relative to that head's vector: a near-zero n . q makes single vectors large (and their rounding with them)
            e = ((y - ref[i]).pow(2).mean(-1).sqrt() / (ref[i].pow(2).mean(-1).sqrt() + 1e-3 * ref[i].pow(2).mean().sqrt())).flatten()
            if kind == seq_ops.STATE_SPACE:
                assert worst_row(y, ref[i]) < 1e-4, i
            else:
                assert float(e.median()) < 1e-5 and float(e.quantile(0.98)) < 2e-3, (i, float(e.median()), float(e.quantile(0.98)))


@pytest.mark.parametrize("rows,groups,size", [(5, 4, 24), (1, 1, 130), (33, 3, 7), (8, 16, 64), (3, 2, 1024), (2, 40, 6)])
@pytest.mark.parametrize("f32", [True, False])
def test_group_norm_and_gates(rows, groups, size, f32):
    from paligemma_multimodal_system_b200 import seq_ops
    dt, D, eps = (torch.float32 if f32 else torch.bfloat16), groups * size, 1e-5
    g = torch.Generator().manual_seed(D)
    o, gate = torch.randn(rows, D, generator=g), torch.randn(rows, D, generator=g).to(torch.bfloat16).float()
    wide, one = torch.randn(D, generator=g), torch.randn(size, generator=g)
    gd = gate.cuda().to(dt)
    buf = torch.full((rows, D + 8), 3.0, device="cuda", dtype=dt)

    def normed(x):
        return O.over_rms(x.view(rows, groups, size), eps).reshape(rows, D)

    for w in (wide, one):
        full = w if w.numel() == D else w.repeat(groups)
        seq_ops.group_norm_gate(o.cuda(), w.cuda(), gd, buf[:, :D], groups, eps, seq_ops.GATE_SIGMOID_AFTER, 0.7)
        assert worst_row(buf[:, :D].float(), 0.7 * normed(o) * full * torch.sigmoid(gate)) < (1e-5 if f32 else 1e-2)
        seq_ops.group_norm_gate(o.cuda(), w.cuda(), gd, buf[:, :D], groups, eps, seq_ops.GATE_SILU_BEFORE)
        assert worst_row(buf[:, :D].float(), normed(o * O.silu(gate)) * full) < (1e-5 if f32 else 1e-2)
        seq_ops.group_norm_gate(o.cuda(), w.cuda(), None, buf[:, :D], groups, eps, seq_ops.GATE_NONE)
        assert worst_row(buf[:, :D].float(), normed(o) * full) < (1e-5 if f32 else 1e-2)
    assert bool((buf[:, D:] == 3.0).all())  # the columns beside the slice are left alone


@pytest.mark.parametrize("rows,D", [(3, 72), (1, 33), (50, 1024), (7, 2052), (2, 5000), (4, 9001)])
@pytest.mark.parametrize("f32", [True, False])
def test_gated_post_norm_residual_and_next_norm(rows, D, f32):
    from paligemma_multimodal_system_b200 import seq_ops
    dt, eps = (torch.float32 if f32 else torch.bfloat16), 1e-5
    g = torch.Generator().manual_seed(D)
    y, x0, gate = 2.0 * torch.randn(rows, D, generator=g) + 1.0, torch.randn(rows, D, generator=g), torch.randn(rows, D, generator=g).to(torch.bfloat16).float()
    gb, w1, b1, w2, b2 = (torch.randn(D, generator=g) for _ in range(5))
    want = x0 + O.layer_norm(y * torch.sigmoid(gate + gb), w1, b1, eps)
    x, out = x0.cuda().contiguous(), torch.empty(rows, D, device="cuda", dtype=dt)
    dev = [t.cuda() for t in (gb, w1, b1, w2, b2)]
    wide = torch.zeros(rows, D + 24, device="cuda", dtype=dt)
    wide[:, 8:8 + D] = gate.cuda().to(dt)
    seq_ops.gated_layernorm_add(y.cuda(), wide[:, 8:8 + D], dev[0], dev[1], dev[2], x, eps, dev[3], dev[4], out)
    assert worst_row(x, want) < 1e-5 and worst_row(out.float(), O.layer_norm(want, w2, b2, eps)) < (1e-5 if f32 else 1e-2)
    x = x0.cuda().contiguous()  # an fp32 gate beside either output type
    seq_ops.gated_layernorm_add(y.cuda(), gate.cuda(), dev[0], dev[1], dev[2], x, eps, dev[3], dev[4], out)
    assert worst_row(x, want) < 1e-5 and worst_row(out.float(), O.layer_norm(want, w2, b2, eps)) < (1e-5 if f32 else 1e-2)
    x = x0.cuda().contiguous()
    seq_ops.gated_layernorm_add(y.cuda(), gate.cuda().to(dt), dev[0], dev[1], dev[2], x, eps)  # the model's last sub-layer: no norm follows
    assert worst_row(x, want) < 1e-5


ATTENTIONS = [dict(), dict(heads=4, kv_heads=1, dim=64, vdim=128, rot_dims=32), dict(heads=6, kv_heads=6, dim=64, vdim=64, rot_dims=64), dict(heads=3, kv_heads=1, dim=10, vdim=7, rot_dims=2),
              dict(heads=8, kv_heads=2, dim=128, vdim=64, rot_dims=8)]


@pytest.mark.parametrize("kw", ATTENTIONS)
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 3e-2)])
def test_logistic_attention_alone(kw, dtype, tol):
    """The attention half of a parallel layer over 200 positions: as one portion, and as context + portion + single tokens (decode kernel)."""
    from paligemma_multimodal_system_b200 import seq_ops
    D, T = 56, 200
    cfg = make_cfg([with_ff(parallel(**kw), 0)], width=D)
    w = O.random_weights(cfg, seed=len(str(kw)))
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(3)).to(torch.bfloat16).float()
    ref = O.logistic_attention(h, w, "l0.mix.left.", cfg["layers"][0]["mixer"]["left"])
    mx = load_mixer(cfg, w).left
    mx.out_scale = 1.0
    prec = seq_ops.Precision(dtype)
    mx.pack(prec)
    for cuts in ([T], [131, 67, 1], [2]):
        assert worst_row(run_mixer(mx, h, cuts, dtype, prec), ref) < tol, cuts


@pytest.mark.parametrize("place", [0, 1, 31, 32, 63, 64, 127, 128, 299])
@pytest.mark.parametrize("dtype,dim,vdim", [(torch.float32, 16, 24), (torch.bfloat16, 64, 64), (torch.bfloat16, 16, 24)])
def test_a_far_key_among_hundreds_stands_out(place, dtype, dim, vdim):
    """One key with a large score and a value of its own at page and tile borders, everything else with a strongly negative bias: dropping
    or doubling it changes the row by its whole size.  Read by a prompt's last row and by a decoded token with many key splits."""
    from paligemma_multimodal_system_b200 import seq_ops
    from paligemma_multimodal_system_b200.cache import SequenceStore
    H, G, n = 4, 2, 300
    g = torch.Generator().manual_seed(place)
    k = 0.1 * torch.randn(n, G, dim, generator=g)
    v = torch.randn(n, G, vdim, generator=g)
    q = torch.ones(n, H, dim)
    k[place] = 1.0
    v[place] = 5.0
    q, k, v = (t.to(torch.bfloat16).float() for t in (q, k, v))
    bias = torch.tensor([-8.0, -9.0, -10.0, -7.5])
    scale = 20.0 / dim
    store = SequenceStore([("kv", G * dim, G * vdim)], max_tokens=448, num_slots=1, dtype=dtype)
    store.k_pages[0].fill_(1e4), store.v_pages[0].fill_(1e4)
    store.pool.take(1)
    store.admit(0)
    rec = store.reserve(0, n)
    for j in range(n):
        store.k_pages[0][rec.pages[j // 64], j % 64] = k[j].reshape(-1).cuda().to(dtype)
        store.v_pages[0][rec.pages[j // 64], j % 64] = v[j].reshape(-1).cuda().to(dtype)
    ref = torch.stack([torch.sigmoid((k[:, h // 2] @ q[-1, h]) * scale + bias[h]) @ v[:, h // 2] for h in range(H)])
    for pitch, osc in ((0, 1.0), (H * vdim + 16, 1.7)):
        score = seq_ops.ScoreOptions(H, logistic=True, head_bias=bias.cuda(), out_scale=osc, out_ld=pitch)
        for first in (0, n - 1):
            b = seq_ops.make_step_batch([dict(tokens=[0] * (n - first), ctx=first, slot=rec.slot, pages=rec.pages)])
            out = torch.zeros(n - first, pitch or H * vdim, device="cuda", dtype=dtype)
            seq_ops.attn_ragged(q[first:].reshape(n - first, -1).cuda().to(dtype).contiguous(), store.k_pages[0], store.v_pages[0], None, out, b, H, G, dim, vdim, scale,
                                0.0, 64, score=score)
            assert worst_row(out[-1, :H * vdim].float().view(H, vdim), osc * ref) < (1e-4 if dtype == torch.float32 else 1e-2), (first, pitch)
            assert not bool(out[:, H * vdim:].any())


MIXERS = [delta(), delta(heads=6, kv_heads=3, dim=64, vdim=32), delta(heads=2, kv_heads=2, dim=40, vdim=64, conv=2), delta(heads=3, kv_heads=1, dim=5, vdim=11, conv=1),
          delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=8),
          parallel(), parallel(heads=4, kv_heads=1, dim=64, vdim=64, rot_dims=32, rheads=4, groups=4, state=64, rvdim=32, norm_groups=2, conv=3),
          parallel(heads=2, kv_heads=2, dim=9, vdim=5, rot_dims=4, rheads=3, groups=1, state=7, rvdim=11, norm_groups=3, conv=1, ls=0.4, rs=2.5),
          memory(), memory(heads=2, dim=48, vdim=64, cap=15.0), memory(heads=4, dim=64, vdim=136, cap=3.0), memory(heads=1, dim=9, vdim=7, cap=1.0)]


def oracle_mixer(l, h, w, eps):
    return O.MIXERS[l["type"]](h, w, "l0.mix.", l["mixer"], eps)


@pytest.mark.parametrize("mi", range(len(MIXERS)))
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-4), (torch.bfloat16, 6e-2)])
def test_mixer_alone_whole_in_portions_and_token_by_token(mi, dtype, tol):
    from paligemma_multimodal_system_b200 import seq_ops
    D, T, eps, l = 56, 140, 1e-5, MIXERS[mi]
    cfg = make_cfg([with_ff(l, 0)], width=D, eps=eps)
    w = O.random_weights(cfg, seed=mi, rank=(9, 16))
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(mi)).to(torch.bfloat16).float()
    ref = oracle_mixer(l, h.double(), {k: v.double() for k, v in w.items()}, eps)
    mx = load_mixer(cfg, w)
    prec = seq_ops.Precision(dtype)
    mx.pack(prec)
    for cuts in ([T], [70, 16, 2, 1], [2], [15, 17]):
        got = run_mixer(mx, h, cuts, dtype, prec)
        if dtype == torch.float32:
            assert worst_row(got, ref) < tol, cuts
        else:
            assert rel_err(got, ref) < tol / 2 and worst_row(got, ref) < 5 * tol, (cuts, rel_err(got, ref), worst_row(got, ref))


def test_side_rows_ride_in_the_input_projection():
    from paligemma_multimodal_system_b200 import seq_ops
    D, T = 56, 30
    prec = seq_ops.Precision(torch.float32)
    for l in (delta(), parallel(), memory()):
        cfg = make_cfg([with_ff(l, 0)], width=D)
        w = O.random_weights(cfg, seed=4)
        h = torch.randn(T, D, generator=torch.Generator().manual_seed(8))
        side = torch.randn(21, D, generator=torch.Generator().manual_seed(9))
        mx = load_mixer(cfg, w)
        mx.pack(prec, side=side)
        store = one_store(mx.cache_specs(), T, torch.float32)
        b = seq_ops.make_step_batch([dict(tokens=[0] * T, ctx=0, slot=store.live[0].slot, pages=store.live[0].pages)])
        y, s = mx(h.cuda(), b, store, 0, prec)
        assert worst_row(s, h @ side.T) < 1e-5 and worst_row(y, oracle_mixer(l, h, w, 1e-5)) < 3e-4


@pytest.mark.parametrize("ff", [80, 33, 256])
@pytest.mark.parametrize("dtype,tol,T", [(torch.float32, 1e-5, 77), (torch.bfloat16, 2e-2, 77), (torch.float32, 1e-5, 1), (torch.bfloat16, 2e-2, 300)])
def test_relu_gated_feed_forward_alone(ff, dtype, tol, T):
    from paligemma_multimodal_system_b200 import seq_ops
    from paligemma_multimodal_system_b200.mixers import GluFeedForward
    D = 64
    w = O.random_weights(make_cfg([with_ff(memory(), ff)], width=D), seed=T)
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16).float()
    f = GluFeedForward(D, ff, "relu")
    left = {k: v.to(torch.bfloat16) for k, v in w.items()}
    f.load(lambda name, shape: left.pop(name), "l0.mlp.")
    prec = seq_ops.Precision(dtype)
    f.pack(prec)
    assert worst_row(f(h.cuda().to(dtype).contiguous(), None, prec), O.feed_forward(h, w, "l0.mlp.")) < tol


def test_a_token_written_long_ago_is_read_back_from_the_state():
    """Slow decays: one token's key is a direction no other key has, and 300 tokens later a query along it must return that token's value."""
    from paligemma_multimodal_system_b200 import seq_ops
    H, dim, vdim, n = 2, 16, 24, 400
    g = torch.Generator().manual_seed(0)
    for mark in (0, 15, 16, 17, 63, 64, 99):
        k = torch.randn(n, H, dim, generator=g)
        k[..., 0] = 0.0
        k[mark] = 0.0
        k[mark, :, 0] = 1.0
        v = torch.randn(n, H, vdim, generator=g)
        q = torch.zeros(n, H, dim)
        q[..., 0] = 1.0
        k, v = k.to(torch.bfloat16).float(), v.to(torch.bfloat16).float()
        for dt in (torch.float32, torch.bfloat16):
            for cuts in ([n], [mark + 1, 1], [100, 2, 298]):
                state = torch.full((1, H, dim, vdim), 1e4, device="cuda")
                pos, i, last = 0, 0, None
                while pos < n:
                    c = min(cuts[min(i, len(cuts) - 1)], n - pos)
                    b = seq_ops.make_step_batch([dict(tokens=[0] * c, ctx=pos, slot=0, pages=list(range((pos + c + 63) // 64)))])
                    part = [t[pos:pos + c].reshape(c, -1).cuda().to(dt).contiguous() for t in (q, k, v)]
                    out = torch.empty(c, H * vdim, device="cuda")
                    beta = torch.full((c, 8), 30.0, device="cuda", dtype=dt)  # writes in full
                    knorm = 1.0 / k[pos:pos + c].norm(dim=-1).cuda()
                    inv = torch.cat([torch.ones(c, H, device="cuda"), knorm], 1).contiguous()
                    seq_ops.delta_rule(*part, beta[:, :H], inv, torch.full((c, H * dim), -20.0, device="cuda"), torch.zeros(H, device="cuda"),
                                       torch.zeros(H * dim, device="cuda"), state, out, b, H, H, dim, vdim)
                    last, pos, i = out[-1].cpu(), pos + c, i + 1
                assert worst_row(last.view(H, vdim), v[mark]) < 1e-3, (mark, dt, cuts)


# ----------------------------------------------------------------------------------------------------------------------
# whole models
# ----------------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def base():
    # weights under which no position divides by a nearly vanishing n . q (bf16 rounding of q and k is amplified there, in any implementation)
    w = O.random_weights(BASE_CFG, seed=2)
    tk = toks(150, BASE_CFG["vocab"], 2)
    return w, tk, O.forward(BASE_CFG, w, tk)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
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
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_portions_and_token_by_token_equal_the_whole_prompt(base, cuts, dtype):
    w, tk, ref = base
    eng = engine_for(BASE_CFG, w, dtype)
    poison(eng)
    assert close(run_cut(eng, "a", tk, cuts), ref, dtype)


def test_causal_edge_and_stale_rows(base):
    """Position i must see row i and not row i + 1: a changed LAST token leaves every earlier position's logits bit-identical."""
    w, _, _ = base
    tk = toks(80, BASE_CFG["vocab"], 6)
    eng = engine_for(BASE_CFG, w, torch.float32)
    poison(eng)
    got = eng.step([("a", tk, list(range(80)))], ["a"])
    tk2 = tk[:-1] + [(tk[-1] + 1) % BASE_CFG["vocab"]]
    got2 = eng.step([("b", tk2, list(range(80)))], ["b"])
    assert torch.equal(got[:-1], got2[:-1]) and not torch.equal(got[-1], got2[-1])
    assert close(got, O.forward(BASE_CFG, w, tk), torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
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


def test_long_decoding_across_page_borders(base):
    w, _, _ = base
    tk = toks(260, BASE_CFG["vocab"], 77)
    ref = O.forward(BASE_CFG, w, tk)
    for dtype in (torch.float32, torch.bfloat16):
        eng = engine_for(BASE_CFG, w, dtype)
        poison(eng)
        assert close(run_cut(eng, "a", tk, [60, 1]), ref, dtype)  # 200 single-token steps: eager, captured, then replayed graphs


def test_first_tokens_of_a_sequence(base):
    """One-token prompts, a one-token first portion, two-token portions from the start."""
    w, tk, ref = base
    eng = engine_for(BASE_CFG, w, torch.float32)
    poison(eng)
    one = eng.step([("x", tk[:1], [0])], ["x"])
    assert close(one, ref[:1], torch.float32)
    assert close(run_cut(eng, "y", tk[:9], [1, 2, 2, 1, 3]), ref[:9], torch.float32)
    assert close(run_cut(eng, "z", tk[:8], [2]), ref[:8], torch.float32)


OTHER_SIZES = [
    # odd sizes the 16-byte paths cannot take, two taps, one head per group, equal and unequal ranks
    make_cfg([with_ff(delta(heads=3, kv_heads=1, dim=10, vdim=7, conv=2), 25), with_ff(parallel(heads=3, kv_heads=3, dim=14, vdim=5, rot_dims=6, rheads=5, groups=5, state=6, rvdim=3, norm_groups=5, conv=2), 0),
              with_ff(memory(heads=2, dim=11, vdim=13, cap=2.0), 25)], width=34, vocab=41),
    # sizes the tensor-core kernels like; a recurrent layer last; eight taps
    make_cfg([with_ff(parallel(heads=4, kv_heads=1, dim=128, vdim=128, rot_dims=64, rheads=4, groups=2, state=128, rvdim=64, norm_groups=2, conv=8), 256),
              with_ff(memory(heads=2, dim=64, vdim=128, cap=20.0), 0), with_ff(delta(heads=4, kv_heads=4, dim=64, vdim=64, conv=8), 128)], width=128, vocab=256, eps=1e-6),
    # a single head everywhere, one tap (no convolution state), values of one column, scales of one
    make_cfg([with_ff(memory(heads=1, dim=1, vdim=1, cap=4.0), 12), with_ff(delta(heads=1, kv_heads=1, dim=2, vdim=1, conv=1), 12),
              with_ff(parallel(heads=1, kv_heads=1, dim=2, vdim=1, rot_dims=2, rheads=1, groups=1, state=1, rvdim=4, norm_groups=1, conv=1, ls=1.0, rs=1.0), 0)], width=24, vocab=20),
]


@pytest.mark.parametrize("ci", range(len(OTHER_SIZES)))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_other_sizes(ci, dtype):
    cfg = OTHER_SIZES[ci]
    w = O.random_weights(cfg, seed=(22, 23, 26)[ci], rank=(5, 8) if ci == 0 else 16)  # well-conditioned: see `base`
    tk = toks(100, cfg["vocab"], ci)
    ref = O.forward(cfg, w, tk)
    eng = engine_for(cfg, w, dtype)
    poison(eng)
    assert close(run_cut(eng, "a", tk, [70, 2, 1, 1, 20, 1]), ref, dtype)
    two = [toks(n, cfg["vocab"], 50 + n) for n in (66, 30)]
    out = eng.step([(i, p, list(range(len(p)))) for i, p in enumerate(two)], [0, 1])
    assert close(out[:66], O.forward(cfg, w, two[0]), dtype) and close(out[66:], O.forward(cfg, w, two[1]), dtype)


GEN_CFG = make_cfg([with_ff(delta(heads=2, kv_heads=2, dim=16, vdim=16), 48), with_ff(parallel(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=8, rheads=2, groups=1, state=16, rvdim=8, norm_groups=2), 32),
                    with_ff(memory(heads=2, dim=8, vdim=16), 0)], width=48, vocab=60)


def test_greedy_generation_through_the_scheduler():
    """engine.generate: more prompts than slots, a pool smaller than the sum of all requests, portions of 48 rows; the tokens
    equal the oracle's greedy continuation of each prompt alone."""
    w = O.random_weights(GEN_CFG, seed=31)
    prompts = [toks(n, 60, 40 + n) for n in (70, 5, 33, 1, 90, 12)]
    new = 10
    eng = engine_for(GEN_CFG, w, torch.float32, max_tokens=5 * 64, slots=3)
    poison(eng)
    got = eng.generate(prompts, new, step_tokens=48)
    for p, g in zip(prompts, got):
        seq = list(p)
        for _ in range(new):
            lg = O.forward(GEN_CFG, w, seq)[-1]
            top2 = lg.topk(2).values
            assert float(top2[0] - top2[1]) > 1e-3, "test weights give a near tie"
            seq.append(int(lg.argmax()))
        assert g == seq[len(p):]
    assert not eng.store.live and len(eng.store.pool.free) == 5


def test_sampled_generation_stays_in_vocabulary_and_stops_at_eos():
    w = O.random_weights(GEN_CFG, seed=9)
    eng = engine_for(GEN_CFG, w, torch.bfloat16, max_tokens=256, slots=2)
    out = eng.generate([toks(20, 60, 1), toks(3, 60, 2), toks(40, 60, 3)], 10, do_sample=True, temperature=0.9, top_p=0.8, eos_token_id=7, seed=3)
    for g in out:
        assert 1 <= len(g) <= 10 and all(0 <= t < 60 for t in g)
        assert 7 not in g[:-1]


def write_checkpoint(path, cfg, w):
    meta, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
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
    eng = SequenceEngine(load_model(str(tmp_path / "m"), dtype=torch.float32), 128, 1)
    assert close(eng.step([("a", tk, list(range(50)))], ["a"]), O.forward(GEN_CFG, w, tk), torch.float32)
    prompts = [toks(5, 60, 45), toks(33, 60, 73)]
    got = inference.main(str(tmp_path / "m"), prompt_ids=";".join(" ".join(map(str, p)) for p in prompts), max_tokens_to_generate=4, dtype="float32")
    for p, g in zip(prompts, got):
        seq = list(p)
        for _ in range(4):
            seq.append(int(O.forward(GEN_CFG, w, seq)[-1].argmax()))
        assert g == seq[len(p):]


def test_wider_model_long_prompt_reaches_the_large_tile_paths():
    """Width 512, a 2048-wide feed-forward and tensor-core head sizes over 1100 tokens in bf16; then 20 decoded tokens."""
    cfg = make_cfg([with_ff(delta(heads=8, kv_heads=8, dim=64, vdim=64), 2048),
                    with_ff(parallel(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=32, rheads=8, groups=2, state=64, rvdim=64, norm_groups=2), 1024),
                    with_ff(memory(heads=4, dim=128, vdim=128), 512)], width=512, vocab=1000)
    w = O.random_weights(cfg, seed=77, rank=64)
    tk = toks(1120, 1000, 3)
    ref = O.forward(cfg, w, tk, dtype=torch.float32)
    eng = engine_for(cfg, w, torch.bfloat16, max_tokens=1280, slots=2)
    poison(eng)
    assert close(run_cut(eng, "a", tk, [1100, 1]), ref, torch.bfloat16)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_a_mixed_schedule(tmp_path, dtype):
    """bin/trace_run on a checkpoint folder: portions beside single tokens, a step that wants nothing, a request that sits out a step,
    a finished request's page and slot taken over by a later one; the written logits equal the oracle's for each request alone."""
    import subprocess
    import numpy as np
    cfg = OTHER_SIZES[0]
    w = O.random_weights(cfg, seed=13, rank=6)
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
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    for step, rows in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        assert close(got, torch.stack([ref[k][p] for k, p in rows]), dt), step
