"""Plain, slow restatement of the Padulorn decoder (test infrastructure only; the product path never imports it).

One function per mechanism, one sequence at a time (positions 0 .. T-1), nothing shared with the kernels or their host wrappers.
x [T, D] is the residual stream, mu one constant of the model, N(z; g) = z / sqrt(mean(z^2) + eps) * g:

    x <- x + mu N(mixer(x); n1);   x <- x + mu N(ff(x); n2)   (layers that have a feed-forward);   logits = c head N(x; nf)

Mixers, each a function of the rows x of one sequence: sliding-window softmax attention that keeps the first tokens visible and blends its
values with an earlier layer's, and retention (a matrix state per head that shrinks by a fixed factor per token).  Feed-forward: routed
experts with logistic scores and a choice limited to the best groups.

A "weights" argument is a dict name -> tensor (any float type) with the checkpoint's names; "cfg" is the parsed config.json.
"""
import math

import torch


def over_rms(z, eps):
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def frequencies(rot):
    """(angle per position of every pair, factor on cosines and sines)."""
    base, dims, sc = float(rot["base"]), int(rot["dims"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0

    def pair_of(turns):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first, last = max(math.floor(pair_of(float(sc["fast"]))), 0), min(math.ceil(pair_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(fi / float(sc["factor"]) * r + fi * (1.0 - r))
    return out, 0.1 * math.log(float(sc["factor"])) + 1.0


def turned(vec, p, rot, partner):
    """vec [..., n] at position p; pair i is (2i, 2i + 1) with partner "next", (i, i + dims / 2) with partner "half"."""
    if not rot or not int(rot.get("dims", 0)):
        return vec
    f, gain = frequencies(rot)
    half, out = len(f), vec.clone()
    for i in range(half):
        a, b = (2 * i, 2 * i + 1) if partner == "next" else (i, i + half)
        c, s = gain * math.cos(p * f[i]), gain * math.sin(p * f[i])
        out[..., a], out[..., b] = vec[..., a] * c - vec[..., b] * s, vec[..., b] * c + vec[..., a] * s
    return out


def visible(i, j, mask):
    if j > i:
        return False
    return not mask or i - j < int(mask["size"]) or j < int(mask.get("keep_first", 0))


def attention(x, w, pre, m, eps, first_values=None):
    """Returns (output, this layer's own values before any blending).  first_values [T, G * vdim]: blend them in by the layer's weight."""
    T = x.shape[0]
    H, G, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = over_rms(x @ w[pre + "q"].T, eps) * w[pre + "q.norm"]
    k = over_rms(x @ w[pre + "k"].T, eps) * w[pre + "k.norm"]
    own = v = x @ w[pre + "v"].T
    if first_values is not None:
        lam = w[pre + "vmix"]
        v = (1.0 - lam) * v + lam * first_values
    rot = m.get("rot")
    q = torch.stack([turned(q[t].view(H, dim), t, rot, "next") for t in range(T)])
    k = torch.stack([turned(k[t].view(G, dim), t, rot, "next") for t in range(T)])
    v = v.view(T, G, vdim)
    out = torch.zeros(T, H, vdim, dtype=x.dtype)
    for i in range(T):
        seen = torch.tensor([j for j in range(i + 1) if visible(i, j, m.get("mask"))])
        for h in range(H):
            g = h // (H // G)
            out[i, h] = torch.softmax((k[seen, g] @ q[i, h]) * float(m["scale"]), 0) @ v[seen, g]
    return out.reshape(T, H * vdim) @ w[pre + "o"].T, own


def retained(q, k, v, decay):
    """q, k [T, H, dim], v [T, H, vdim], decay [H]: S <- decay S + k v^T, o = S^T q, per head, token by token."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(x, w, pre, m, eps):
    T = x.shape[0]
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    rot = m.get("rot")
    q, k, v = (x @ w[pre + n].T for n in "qkv")
    q = torch.stack([turned(q[t].view(H, dim), t, rot, "half") for t in range(T)])
    k = torch.stack([turned(k[t].view(H, dim), t, rot, "half") for t in range(T)]) * dim ** -0.5
    o = over_rms(retained(q, k, v.view(T, H, vdim), torch.tensor(m["decay"], dtype=x.dtype)), eps)
    return (o.reshape(T, H * vdim) * silu(x @ w[pre + "g"].T)) @ w[pre + "o"].T


def chosen(z, router):
    """Router outputs of one token -> [(expert, weight)]."""
    s = torch.sigmoid(z)
    n, groups = int(router["experts"]), router.get("groups")
    allowed = range(n)
    if groups:
        count, size = int(groups["count"]), n // int(groups["count"])
        score = [float(s[g * size:(g + 1) * size].sort(descending=True).values[:2].sum()) for g in range(count)]
        best = sorted(range(count), key=lambda g: (-score[g], g))[:int(groups["keep"])]
        allowed = [e for e in range(n) if e // size in best]
    return [(e, s[e]) for e in sorted(allowed, key=lambda e: (-float(s[e]), e))[:int(router["top"])]]


def experts(x, w, pre, mlp):
    out = torch.zeros_like(x)
    z = x @ w[pre + "router"].T
    for t in range(x.shape[0]):
        for e, weight in chosen(z[t], mlp["router"]):
            out[t] += weight * (w[f"{pre}e{e}.down"] @ gelu_erf(w[f"{pre}e{e}.up"] @ x[t]))
    return out


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps, mu = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    layers, first = [], None
    for i, l in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", l["mixer"]
        if l["type"] == "attention":
            y, own = attention(x, w, pre + "mix.", m, eps, first if m.get("v_mix") else None)
            if m.get("v_mix") and first is None:
                first = own
        else:
            y = retention(x, w, pre + "mix.", m, eps)
        x = x + mu * over_rms(y, eps) * w[pre + "norm1"]
        if l.get("mlp"):
            x = x + mu * over_rms(experts(x, w, pre + "mlp.", l["mlp"]), eps) * w[pre + "norm2"]
        layers.append(x.clone())
    logits = (over_rms(x, eps) * w["final.norm"]) @ w["head"].T * float(cfg["logit_scale"])
    return (logits, layers) if return_layers else logits


def tensor_shapes(cfg):
    D, V = int(cfg["width"]), int(cfg["vocab"])
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        x = p + "mix."
        H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        G = int(m["kv_heads"]) if l["type"] == "attention" else H
        s.update({p + "norm1": (D,), x + "q": (H * dim, D), x + "k": (G * dim, D), x + "v": (G * vdim, D), x + "o": (D, H * vdim)})
        if l["type"] == "attention":
            s.update({x + "q.norm": (H * dim,), x + "k.norm": (G * dim,)})
            if m.get("v_mix"):
                s[x + "vmix"] = ()
        else:
            s[x + "g"] = (H * vdim, D)
        if l.get("mlp"):
            F, n = int(l["mlp"]["expert"]["ff"]), int(l["mlp"]["router"]["experts"])
            s.update({p + "norm2": (D,), p + "mlp.router": (n, D)})
            for e in range(n):
                s.update({f"{p}mlp.e{e}.up": (F, D), f"{p}mlp.e{e}.down": (D, F)})
    return s


def random_weights(cfg, seed=0):
    """bf16-representable random weights that keep activations near one."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith("vmix"):
            t = 0.45 + 0.1 * r
        elif name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r / float(cfg["embedding"]["scale"])
        else:
            t = r * (1.3 / math.sqrt(shape[-1]))
        w[name] = t.to(torch.bfloat16).float()
    return w
