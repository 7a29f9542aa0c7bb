"""Fadosun: a decoder-only language model of gated sub-layers with a norm before and after each, most of whose layers carry a recurrent
matrix state instead of keys and values, served through the ragged-step engine (engine.py).

    a = LN(x; n1);   x <- x + LN(mixer(a) * sigmoid(R1 a + r1); n1')
    a = LN(x; n2);   x <- x + LN(ff(a)    * sigmoid(R2 a + r2); n2')         (layers that have a feed-forward)
    logits = head LN(x; nf)

LN = layer norm with weight and bias.  Mixer types of a config:

    channel_delta  `mixers.ChannelDeltaRule`: delta rule with one decay per head and key channel, behind short convolutions
    parallel       `mixers.SideBySide`: logistic attention (`mixers.LogisticAttention`) beside a state-space recurrence
                   (`mixers.StateSpaceMixer`), a weighted sum
    mlstm          `mixers.MatrixMemory`: exponentially gated matrix memory

Feed-forward "dense": relu-gated (`mixers.GluFeedForward`).

Every size and model-dependent constant comes from config.json (`FadosunConfig`) or a tensor's shape, tensor names from the checkpoint:

    embed, final.norm{,.b}, head, l<i>.{norm1,norm1b,norm2,norm2b}{,.b}, l<i>.{rg1,rg2}{,.b}, l<i>.mlp.{gate,up,down},
    l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,A_log,norm,a1,a2,dt_bias,g1,g2,o} (channel_delta), l<i>.mix.left.{q,k,v,pb,o} and
    l<i>.mix.right.{in,conv,conv.b,dt_bias,A_log,D,norm,o} (parallel), l<i>.mix.{q,k,v,g,o,norm,i,i.b,f,f.b} (mlstm)

A layer owns a run of store entries, in the order of its mixer's `cache_specs()`.  The residual stream is fp32; one kernel per
sub-layer gates its result, normalises it, adds it and forms the next sub-layer's input (seq_ops.gated_layernorm_add).  The gate R1 a of
a mixer comes from the mixer's own input projection.
"""
import json
import os
from typing import Dict, List, Optional

import torch

from . import _lib, seq_ops
from .mixers import ChannelDeltaRule, GluFeedForward, LogisticAttention, MatrixMemory, SideBySide, StateSpaceMixer

MIXER_TYPES = ("channel_delta", "parallel", "mlstm")


class FadosunConfig:
    def __init__(self, cfg: dict):
        if cfg.get("architecture") != "Fadosun":
            raise ValueError("not a Fadosun config")
        self.raw = cfg
        self.vocab = int(cfg["vocab"])
        self.width = int(cfg["width"])
        self.norm_eps = float(cfg["norm"]["eps"])
        self.layers: List[dict] = list(cfg["layers"])
        for i, l in enumerate(self.layers):
            if l["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            if l.get("mlp") and l["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp'].get('kind')!r}")

    @classmethod
    def from_dir(cls, path):
        with open(os.path.join(path, "config.json")) as f:
            return cls(json.load(f))


def _mixer(width: int, kind: str, m: dict, eps: float):
    if kind == "channel_delta":
        return ChannelDeltaRule(width, int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m.get("vdim", m["dim"])), int(m["conv"]), eps)
    if kind == "mlstm":
        return MatrixMemory(width, int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), m["gate_cap"], eps)
    l, r = m["left"], m["right"]
    rot = l.get("rot") or {}
    left = LogisticAttention(width, int(l["heads"]), int(l.get("kv_heads", l["heads"])), int(l["dim"]), int(l.get("vdim", l["dim"])), l["scale"],
                             int(rot.get("dims", 0)), rot.get("base", 10000.0))
    right = StateSpaceMixer(width, int(r["heads"]), int(r.get("groups", 1)), int(r["state"]), int(r["vdim"]), int(r["conv"]), int(r.get("norm_groups", 1)), eps)
    return SideBySide(left, right, m.get("left_scale", 1.0), m.get("right_scale", 1.0))


class GatedSublayer:
    """The norms and the result gate around one sub-layer: names norm<n>, norm<n>b, rg<n> (each with a bias `.b`)."""

    def __init__(self, n, width):
        self.n, self.D = n, width

    def load(self, take, p):
        D, n = self.D, self.n
        self.w = {k: take(f"{p}{name}", shape) for k, name, shape in (
            ("pre", f"norm{n}", (D,)), ("pre_b", f"norm{n}.b", (D,)), ("post", f"norm{n}b", (D,)), ("post_b", f"norm{n}b.b", (D,)), ("rg", f"rg{n}", (D, D)),
            ("rg_b", f"rg{n}.b", (D,)))}

    def pack(self, prec):
        f32 = dict(device="cuda", dtype=torch.float32)
        self.pre, self.pre_b, self.post, self.post_b, self.rg_b = (self.w[k].to(**f32).contiguous() for k in ("pre", "pre_b", "post", "post_b", "rg_b"))
        self.rg = self.w["rg"].to("cuda", prec.dtype).contiguous()


class FadosunBlock:
    def __init__(self, c: FadosunConfig, i: int):
        l = c.layers[i]
        self.i = i
        self.mixer = _mixer(c.width, l["type"], l["mixer"], c.norm_eps)
        self.sub1 = GatedSublayer(1, c.width)
        self.ff = GluFeedForward(c.width, int(l["mlp"]["ff"]), "relu") if l.get("mlp") else None
        self.sub2 = GatedSublayer(2, c.width) if self.ff is not None else None

    def load(self, take):
        p = f"l{self.i}."
        self.sub1.load(take, p)
        self.mixer.load(take, p + "mix.")
        if self.ff is not None:
            self.sub2.load(take, p)
            self.ff.load(take, p + "mlp.")

    def pack(self, prec):
        self.sub1.pack(prec)
        self.mixer.pack(prec, side=self.sub1.w["rg"])
        if self.ff is not None:
            self.sub2.pack(prec)
            self.ff.pack(prec)


class FadosunForCausalLM:
    """Weights + the step function.  `step(batch, store, want_rows)` advances every entry of a ragged batch by its new tokens (keys, values,
    recurrent and convolution states are left in `store`) and returns fp32 logits of the wanted rows."""

    architecture = "Fadosun"

    def __init__(self, config: FadosunConfig, dtype: torch.dtype = torch.bfloat16):
        self.config = config
        self.prec = seq_ops.Precision(dtype)
        self.blocks = [FadosunBlock(config, i) for i in range(len(config.layers))]
        self.vocab_size = config.vocab
        self._packed = False
        self.cache_at, at = [], 0
        for blk in self.blocks:
            self.cache_at.append(at)
            at += len(blk.mixer.cache_specs())

    # -- weights -------------------------------------------------------------------------------------------------------
    def load_weights(self, tensors: Dict[str, torch.Tensor]):
        """Every tensor must be used and have the shape the config implies (None in a shape: the checkpoint decides); anything missing or
        left over raises."""
        c = self.config
        left = dict(tensors)

        def take(name, shape):
            if name not in left:
                raise KeyError(f"checkpoint lacks {name}")
            t = left.pop(name)
            if t.dim() != len(shape) or any(n is not None and n != m for n, m in zip(shape, t.shape)):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, config implies {tuple(shape)}")
            return t

        self.embed = take("embed", (c.vocab, c.width))
        for blk in self.blocks:
            blk.load(take)
        self.final_norm, self.final_norm_b = take("final.norm", (c.width,)), take("final.norm.b", (c.width,))
        self.head = take("head", (c.vocab, c.width))
        for blk in self.blocks:  # a layer without a feed-forward has no second sub-layer; norms and gate a checkpoint kept for it are unused
            if blk.ff is None:
                for name in ("norm2", "norm2.b", "norm2b", "norm2b.b", "rg2", "rg2.b"):
                    left.pop(f"l{blk.i}.{name}", None)
        if left:
            raise KeyError(f"checkpoint tensors without a place in the model: {sorted(left)[:8]}")
        self._packed = False
        return self

    def pack(self):
        _lib.require_device()
        dt = self.prec.dtype
        self.embed_d = self.embed.to("cuda", dt).contiguous()
        self.final_d = self.final_norm.to("cuda", torch.float32).contiguous()
        self.final_bd = self.final_norm_b.to("cuda", torch.float32).contiguous()
        self.head_d = self.head.to("cuda", dt).contiguous()
        for blk in self.blocks:
            blk.pack(self.prec)
        torch.cuda.synchronize()
        self._packed = True

    def cache_layout(self):
        """The layers' store entries one after the other; layer i's start at cache_at[i]."""
        return [spec for blk in self.blocks for spec in blk.mixer.cache_specs()]

    # -- compute -------------------------------------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, b: seq_ops.StepBatch, store, want_rows: Optional[torch.Tensor], trace: Optional[list] = None):
        """want_rows: int64 row indices (device) whose logits are returned as fp32 [n, vocab]; None / empty: no head."""
        if not self._packed:
            self.pack()
        c, prec, eps = self.config, self.prec, self.config.norm_eps
        x = seq_ops.embed_rows(b.tokens, self.embed_d, 0, c.width, 1.0)
        subs = [s for blk in self.blocks for s in (blk.sub1, blk.sub2) if s is not None]
        following = dict(zip(map(id, subs), subs[1:]))
        a = prec.empty(b.T, c.width)
        if subs:
            seq_ops.layernorm_shift(x, subs[0].pre, subs[0].pre_b, a, eps)

        def join(sub, y, gate):
            """x += post-norm of the gated result; a = what the next sub-layer reads."""
            nxt = following.get(id(sub))
            seq_ops.gated_layernorm_add(y, gate, sub.rg_b, sub.post, sub.post_b, x, eps, *((nxt.pre, nxt.pre_b, a) if nxt is not None else ()))

        for li, blk in enumerate(self.blocks):
            join(blk.sub1, *blk.mixer(a, b, store, self.cache_at[li], prec))
            if blk.ff is not None:
                # few rows: an fp32 product may split its reduction over the whole GPU
                gate = seq_ops.linear(a, blk.sub2.rg, torch.empty(b.T, c.width, device="cuda", dtype=torch.float32 if b.T <= 128 else prec.dtype))
                join(blk.sub2, blk.ff(a, b, prec), gate)
            if trace is not None:
                trace.append(x.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        last = x.index_select(0, want_rows)
        hn = prec.empty(*last.shape)
        seq_ops.layernorm_shift(last, self.final_d, self.final_bd, hn, eps)
        return seq_ops.linear(hn, self.head_d, torch.empty(last.shape[0], c.vocab, device="cuda", dtype=torch.float32))


def load_fadosun(path: str, dtype: torch.dtype = torch.bfloat16) -> FadosunForCausalLM:
    from .utils import read_safetensors
    model = FadosunForCausalLM(FadosunConfig.from_dir(path), dtype)
    return model.load_weights(read_safetensors(os.path.join(path, "model.safetensors")))
