"""Padulorn: a decoder-only language model whose sub-layers read the residual itself and carry their norm on the output, mixing tokens by
windowed softmax attention or by retention, with routed experts, served through the ragged-step engine (engine.py).

    x <- x + mu N(mixer(x)) n1;   x <- x + mu N(ff(x)) n2   (layers that have a feed-forward)
    logits = c head (N(x) nf)                               N(z) = z / sqrt(mean(z^2) + eps);  mu, c: config constants

Mixer types of a config:

    attention  `mixers.WindowedSoftmaxAttention`: q/k norms over the whole projections, partial interleaved rotation with ramped
               frequencies, a sliding window that keeps the first tokens, values blended with those of the first blending layer
    retention  `mixers.Retention`: fixed-decay linear attention with rotated queries and keys, per-head output norm, silu gate

Feed-forward "moe": `mixers.RoutedFeedForward` with erf-gelu experts, logistic scores used as weights as they are, groups ranked by their
two best scores.

Every size and model-dependent constant comes from config.json (`PadulornConfig`), tensor names from the checkpoint:

    embed, final.norm, head, l<i>.{norm1,norm2}, l<i>.mix.{q,k,v,o,q.norm,k.norm,vmix} (attention), l<i>.mix.{q,k,v,g,o} (retention),
    l<i>.mlp.{router,e<k>.up,e<k>.down}

The residual stream is fp32.  mu is folded into the fp32 norm weights and c into the final one; norm, residual add and the activation-type copy
the next product reads are one kernel per sub-layer (behind experts the combine is part of it too).
"""
import json
import os
from typing import Dict, List, Optional

import torch

from . import _lib, seq_ops
from .mixers import Retention, RoutedFeedForward, WindowedSoftmaxAttention

MIXER_TYPES = ("attention", "retention")


class PadulornConfig:
    def __init__(self, cfg: dict):
        if cfg.get("architecture") != "Padulorn":
            raise ValueError("not a Padulorn config")
        self.raw = cfg
        self.vocab = int(cfg["vocab"])
        self.width = int(cfg["width"])
        self.embedding_scale = float((cfg.get("embedding") or {}).get("scale", 1.0))
        self.logit_scale = float(cfg.get("logit_scale", 1.0))
        self.residual_mult = float(cfg.get("residual_mult", 1.0))
        self.norm_eps = float(cfg["norm"]["eps"])
        self.layers: List[dict] = list(cfg["layers"])
        blending = []
        for i, l in enumerate(self.layers):
            if l["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            if l.get("mlp") and l["mlp"].get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp'].get('kind')!r}")
            if l["type"] == "attention" and l["mixer"].get("v_mix"):
                m = l["mixer"]
                blending.append((i, int(m.get("kv_heads", m["heads"])) * int(m.get("vdim", m["dim"]))))
        for i, size in blending[1:]:
            if size != blending[0][1]:
                raise ValueError(f"layer {i}: {size} value elements a token, but layer {blending[0][0]}, whose values it blends in, has {blending[0][1]}")
        self.first_blending = blending[0][0] if blending else None

    @classmethod
    def from_dir(cls, path):
        with open(os.path.join(path, "config.json")) as f:
            return cls(json.load(f))


def _mixer(c: PadulornConfig, i: int):
    kind, m = c.layers[i]["type"], c.layers[i]["mixer"]
    rot = m.get("rot") or {}
    heads, dim = int(m["heads"]), int(m["dim"])
    vdim, dims, base = int(m.get("vdim", dim)), int(rot.get("dims", 0)), rot.get("base", 10000.0)
    if kind == "retention":
        if rot.get("scaling"):
            raise ValueError(f"layer {i}: retention turns with plain frequencies")
        return Retention(c.width, heads, dim, vdim, m["decay"], c.norm_eps, dims, base, rot_layout="half")
    mask = m.get("mask") or {}
    return WindowedSoftmaxAttention(c.width, heads, int(m.get("kv_heads", heads)), dim, vdim, m["scale"], c.norm_eps, window=mask.get("size"),
                                    keep_first=int(mask.get("keep_first", 0)), qk_norm="projection", rot_dims=dims, rot_base=base,
                                    rot_scaling=rot.get("scaling"),
                                    value_blend=None if not m.get("v_mix") else "first" if i == c.first_blending else "later")


def _feed_forward(width: int, mlp: Optional[dict]):
    if not mlp:
        return None
    r = mlp["router"]
    groups = r.get("groups") or {}
    count = int(groups.get("count", 1))
    return RoutedFeedForward(width, int(r["experts"]), 0, int(r["top"]), count, int(groups.get("keep", count)), 1.0, int(mlp["expert"]["ff"]), 0,
                             activation="gelu", correction=False, scores="logistic", group_best=2, normalize=False)


class PadulornBlock:
    def __init__(self, c: PadulornConfig, i: int):
        self.i, self.D, self.mult = i, c.width, c.residual_mult
        self.mixer = _mixer(c, i)
        self.ff = _feed_forward(c.width, c.layers[i].get("mlp"))

    def load(self, take):
        p = f"l{self.i}."
        self.norm1 = take(p + "norm1", (self.D,))
        self.mixer.load(take, p + "mix.")
        if self.ff is not None:
            self.norm2 = take(p + "norm2", (self.D,))
            self.ff.load(take, p + "mlp.")

    def pack(self, prec):
        self.norm1_d = (self.mult * self.norm1.to("cuda", torch.float32)).contiguous()
        self.mixer.pack(prec)
        if self.ff is not None:
            self.norm2_d = (self.mult * self.norm2.to("cuda", torch.float32)).contiguous()
            self.ff.pack(prec)


class PadulornForCausalLM:
    """Weights + the step function.  `step(batch, store, want_rows)` advances every entry of a ragged batch by its new tokens (keys, values and
    recurrent states are left in `store`) and returns fp32 logits of the wanted rows."""

    architecture = "Padulorn"

    def __init__(self, config: PadulornConfig, dtype: torch.dtype = torch.bfloat16):
        self.config = config
        self.prec = seq_ops.Precision(dtype)
        self.blocks = [PadulornBlock(config, i) for i in range(len(config.layers))]
        self.vocab_size = config.vocab
        self._packed = False

    # -- weights -------------------------------------------------------------------------------------------------------
    def load_weights(self, tensors: Dict[str, torch.Tensor]):
        """Every tensor must be used and have the shape the config implies; anything missing or left over raises."""
        c = self.config
        left = dict(tensors)

        def take(name, shape):
            if name not in left:
                raise KeyError(f"checkpoint lacks {name}")
            t = left.pop(name)
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, config implies {tuple(shape)}")
            return t

        self.embed = take("embed", (c.vocab, c.width))
        for blk in self.blocks:
            blk.load(take)
        self.final_norm = take("final.norm", (c.width,))
        self.head = take("head", (c.vocab, c.width))
        for blk in self.blocks:  # what a checkpoint kept for parts a layer does not have
            if blk.ff is None:
                left.pop(f"l{blk.i}.norm2", None)
            left.pop(f"l{blk.i}.mix.vmix", None)
        if left:
            raise KeyError(f"checkpoint tensors without a place in the model: {sorted(left)[:8]}")
        self._packed = False
        return self

    def pack(self):
        _lib.require_device()
        dt = self.prec.dtype
        self.embed_d = self.embed.to("cuda", dt).contiguous()
        self.final_norm_d = (self.config.logit_scale * self.final_norm.to("cuda", torch.float32)).contiguous()
        self.head_d = self.head.to("cuda", dt).contiguous()
        for blk in self.blocks:
            blk.pack(self.prec)
        torch.cuda.synchronize()
        self._packed = True

    def cache_layout(self):
        """One store entry per layer: key / value pages or a state slot."""
        return [spec for blk in self.blocks for spec in blk.mixer.cache_specs()]

    # -- compute -------------------------------------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, b: seq_ops.StepBatch, store, want_rows: Optional[torch.Tensor], trace: Optional[list] = None):
        """want_rows: int64 row indices (device) whose logits are returned as fp32 [n, vocab]; None / empty: no head."""
        if not self._packed:
            self.pack()
        c, prec, eps = self.config, self.prec, self.config.norm_eps
        b = seq_ops.step_scope(b)
        # the sub-layers read x in the activation type: in fp32 that is x itself, in bf16 a rounded copy each residual kernel leaves
        copy = None if prec.f32 else prec.empty(b.T, c.width)
        x = seq_ops.embed_rows(b.tokens, self.embed_d, 0, c.width, c.embedding_scale, out_act=copy)
        xa = x if copy is None else copy
        for li, blk in enumerate(self.blocks):
            y = blk.mixer(xa, b, store, li, prec)
            seq_ops.group_rmsnorm_add(y, blk.norm1_d, x, copy, 1, eps)
            if blk.ff is not None:
                blk.ff.add_normed(xa, prec, blk.norm2_d, x, copy, eps)
            if trace is not None:
                trace.append(x.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        last = x.index_select(0, want_rows)
        hn = prec.empty(*last.shape)
        seq_ops.group_rmsnorm_add(last, self.final_norm_d, None, hn, 1, eps)
        return seq_ops.linear(hn, self.head_d, torch.empty(last.shape[0], c.vocab, device="cuda", dtype=torch.float32))


def load_padulorn(path: str, dtype: torch.dtype = torch.bfloat16) -> PadulornForCausalLM:
    from .utils import read_safetensors
    model = PadulornForCausalLM(PadulornConfig.from_dir(path), dtype)
    return model.load_weights(read_safetensors(os.path.join(path, "model.safetensors")))
