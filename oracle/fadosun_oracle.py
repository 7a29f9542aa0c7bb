"""Plain, slow restatement of the Fadosun decoder (test infrastructure only; the product path never imports it).

One function per mechanism, one sequence at a time (positions 0 .. T-1), nothing shared with the kernels or their host wrappers.
For a layer with residual x [T, D]:

    a = LN(x; norm1);   x <- x + LN(mixer(a) * sigmoid(R1 a + r1); norm1b)
    a = LN(x; norm2);   x <- x + LN(ff(a)    * sigmoid(R2 a + r2); norm2b)          (layers that have a feed-forward)

Mixers, each a function of the rows a of one sequence: the per-channel-decay delta rule (behind short convolutions), unnormalised
logistic attention and the scalar-decay state-space recurrence side by side, and the exponentially gated matrix memory.

A "weights" argument is a dict name -> tensor (any float type) with the checkpoint's names; "cfg" is the parsed config.json.
"""
import math

import torch


def layer_norm(x, g, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * g + b


def over_rms(z, eps):
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def short_conv(u, w, b=None):
    """u [T, C], w [C, taps]: y_t[c] = sum_j w[c, j] u_{t - (taps - 1) + j}[c] (+ b[c]); u before the start is zero."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = sum(w[:, j] * padded[j:j + T] for j in range(taps))
    return y if b is None else y + b


def unit(z):
    return z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k [T, H, dim], v [T, H, vdim], beta [T, H], g [T, H, dim]; S [dim, vdim] per head, rows decayed by g before the write."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_delta(a, w, pre, m, eps):
    T = a.shape[0]
    H, G, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(short_conv(a @ w[pre + n].T, w[pre + n + ".conv"])) for n in "qkv")
    pick = torch.arange(H) // (H // G)
    q = (unit(q.view(T, G, dim)) * dim ** -0.5)[:, pick]
    k = unit(k.view(T, G, dim))[:, pick]
    beta = torch.sigmoid(a @ w[pre + "b"].T)
    z = softplus((a @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]).view(T, H, dim)
    g = torch.exp(-torch.exp(w[pre + "A_log"])[:, None] * z)
    o = delta_rule(q, k, v.view(T, H, vdim), beta, g)
    gate = torch.sigmoid((a @ w[pre + "g1"].T) @ w[pre + "g2"].T)
    return ((over_rms(o, eps) * w[pre + "norm"]).reshape(T, H * vdim) * gate) @ w[pre + "o"].T


def turn_half(vec, p, base, dims):
    """vec [..., n]: element i of the first half of the first `dims` is paired with element i + dims / 2."""
    half, out = dims // 2, vec.clone()
    for i in range(half):
        angle = p * float(base) ** (-2.0 * i / dims)
        c, s = math.cos(angle), math.sin(angle)
        u, v = vec[..., i], vec[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def logistic_attention(a, w, pre, m):
    T = a.shape[0]
    H, G, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (a @ w[pre + n].T for n in "qkv")
    q, k, v = q.view(T, H, dim), k.view(T, G, dim), v.view(T, G, vdim)
    base, dims = m["rot"]["base"], int(m["rot"]["dims"])
    q = torch.stack([turn_half(q[t], t, base, dims) for t in range(T)])
    k = torch.stack([turn_half(k[t], t, base, dims) for t in range(T)])
    out = torch.zeros(T, H, vdim, dtype=a.dtype)
    for i in range(T):
        for h in range(H):
            g = h // (H // G)
            p = torch.sigmoid((k[:i + 1, g] @ q[i, h]) * float(m["scale"]) + w[pre + "pb"][h])
            out[i, h] = p @ v[:i + 1, g]
    return out.reshape(T, H * vdim) @ w[pre + "o"].T


def state_space(x, B, C, dt, decay_rate):
    """x [T, H, vdim], B, C [T, H, N] (already per head), dt [T, H]; S <- exp(-rate dt) S + dt B x^T, y = S^T C."""
    T, H, vdim = x.shape
    S = torch.zeros(H, B.shape[-1], vdim, dtype=x.dtype)
    out = []
    for t in range(T):
        S = torch.exp(-decay_rate * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, C[t]))
    return torch.stack(out)


def state_space_mixer(a, w, pre, m, eps):
    T = a.shape[0]
    H, G, N, vdim, parts = int(m["heads"]), int(m["groups"]), int(m["state"]), int(m["vdim"]), int(m["norm_groups"])
    inner = H * vdim
    z, xbc, dt = torch.split(a @ w[pre + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    pick = torch.arange(H) // (H // G)
    x = x.reshape(T, H, vdim)
    y = state_space(x, B.reshape(T, G, N)[:, pick], C.reshape(T, G, N)[:, pick], softplus(dt + w[pre + "dt_bias"]), torch.exp(w[pre + "A_log"]))
    y = (y + w[pre + "D"][:, None] * x).reshape(T, inner) * silu(z)
    y = over_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def parallel_mixer(a, w, pre, m, eps):
    return (float(m["left_scale"]) * logistic_attention(a, w, pre + "left.", m["left"])
            + float(m["right_scale"]) * state_space_mixer(a, w, pre + "right.", m["right"], eps))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, dim], v [T, H, vdim]; i, f [T, H] log gates.  The running maximum starts at 0."""
    T, H, dim = q.shape
    S, n, top = torch.zeros(H, dim, v.shape[-1], dtype=q.dtype), torch.zeros(H, dim, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, put = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(a, w, pre, m, eps):
    T = a.shape[0]
    H, dim, vdim, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (a @ w[pre + "q"].T).view(T, H, dim) * dim ** -0.5
    k = (a @ w[pre + "k"].T).view(T, H, dim)
    v = (a @ w[pre + "v"].T).view(T, H, vdim)
    i = cap * torch.tanh((a @ w[pre + "i"].T + w[pre + "i.b"]) / cap)
    f = -softplus(-cap * torch.tanh((a @ w[pre + "f"].T + w[pre + "f.b"]) / cap))
    o = over_rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * vdim)
    return (o * w[pre + "norm"] * torch.sigmoid(a @ w[pre + "g"].T)) @ w[pre + "o"].T


def feed_forward(a, w, pre):
    return (torch.relu(a @ w[pre + "gate"].T) * (a @ w[pre + "up"].T)) @ w[pre + "down"].T


MIXERS = {"channel_delta": channel_delta, "parallel": parallel_mixer, "mlstm": mlstm}


def sublayer(x, w, pre, n, fn, eps):
    a = layer_norm(x, w[f"{pre}norm{n}"], w[f"{pre}norm{n}.b"], eps)
    y = fn(a) * torch.sigmoid(a @ w[f"{pre}rg{n}"].T + w[f"{pre}rg{n}.b"])
    return x + layer_norm(y, w[f"{pre}norm{n}b"], w[f"{pre}norm{n}b.b"], eps)


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    layers = []
    for i, l in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = sublayer(x, w, pre, 1, lambda a: MIXERS[l["type"]](a, w, pre + "mix.", l["mixer"], eps), eps)
        if l.get("mlp"):
            x = sublayer(x, w, pre, 2, lambda a: feed_forward(a, w, pre + "mlp."), eps)
        layers.append(x.clone())
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    return (logits, layers) if return_layers else logits


def tensor_shapes(cfg, rank=12):
    """rank: inner width of the two low-rank projections of a channel_delta mixer (a checkpoint says it by its shapes only); a pair
    (decay rank, gate rank) when they differ."""
    D, V = int(cfg["width"]), int(cfg["vocab"])
    ra, rg = rank if isinstance(rank, tuple) else (rank, rank)
    s = {"embed": (V, D), "final.norm": (D,), "final.norm.b": (D,), "head": (V, D)}

    def sub(p, n):
        s.update({f"{p}norm{n}": (D,), f"{p}norm{n}.b": (D,), f"{p}norm{n}b": (D,), f"{p}norm{n}b.b": (D,), f"{p}rg{n}": (D, D), f"{p}rg{n}.b": (D,)})

    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        sub(p, 1)
        x = p + "mix."
        if l["type"] == "channel_delta":
            H, G, dim, vdim, taps = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
            s.update({x + "q": (G * dim, D), x + "q.conv": (G * dim, taps), x + "k": (G * dim, D), x + "k.conv": (G * dim, taps), x + "v": (H * vdim, D),
                      x + "v.conv": (H * vdim, taps), x + "b": (H, D), x + "A_log": (H,), x + "norm": (vdim,), x + "a1": (ra, D), x + "a2": (H * dim, ra),
                      x + "dt_bias": (H * dim,), x + "g1": (rg, D), x + "g2": (H * vdim, rg), x + "o": (D, H * vdim)})
        elif l["type"] == "parallel":
            le, ri = m["left"], m["right"]
            H, G, dim, vdim = (int(le[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            s.update({x + "left.q": (H * dim, D), x + "left.k": (G * dim, D), x + "left.v": (G * vdim, D), x + "left.pb": (H,), x + "left.o": (D, H * vdim)})
            H, G, N, vdim, taps = (int(ri[k]) for k in ("heads", "groups", "state", "vdim", "conv"))
            inner = H * vdim
            C = inner + 2 * G * N
            s.update({x + "right.in": (inner + C + H, D), x + "right.conv": (C, taps), x + "right.conv.b": (C,), x + "right.dt_bias": (H,),
                      x + "right.A_log": (H,), x + "right.D": (H,), x + "right.norm": (inner,), x + "right.o": (D, inner)})
        else:
            H, dim, vdim = (int(m[k]) for k in ("heads", "dim", "vdim"))
            s.update({x + "q": (H * dim, D), x + "k": (H * dim, D), x + "v": (H * vdim, D), x + "g": (H * vdim, D), x + "o": (D, H * vdim),
                      x + "norm": (H * vdim,), x + "i": (H, D), x + "i.b": (H,), x + "f": (H, D), x + "f.b": (H,)})
        if l.get("mlp"):
            sub(p, 2)
            F = int(l["mlp"]["ff"])
            s.update({p + "mlp.gate": (F, D), p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    return s


def random_weights(cfg, seed=0, rank=12):
    """bf16-representable random weights of a size that keeps activations near one; decays from fast to slow, gates of both signs."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        r = torch.randn(shape, generator=g)
        if name.endswith(".A_log"):
            t = torch.rand(shape, generator=g) * 2.5 - 2.0
        elif name.endswith("dt_bias"):
            t = torch.rand(shape, generator=g) * 4.0 - 4.0
        elif name.endswith(".f.b"):
            t = 2.0 + 1.5 * r
        elif name.endswith(".pb"):
            t = -2.0 + 0.5 * r
        elif name.endswith((".b", ".D")) and len(shape) == 1:
            t = 0.3 * r
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1.0 + 0.2 * r
        elif name.endswith(".conv"):
            t = r * 0.6
        elif name == "embed":
            t = r
        else:
            t = r * (1.3 / math.sqrt(shape[-1]))
        w[name] = t.to(torch.bfloat16).float()
    return w
