"""Host-side parts of the Padulorn decoder (configuration, weight accounting, cache layout, registry) and the oracle against itself; no GPU."""
import json
import math
import os
import struct
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from oracle import padulorn_oracle as O  # noqa: E402


def cfg_small():
    att = {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "scale": 0.4, "v_mix": True, "mask": {"size": 7, "keep_first": 3},
           "rot": {"base": 500.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}}
    ret = {"heads": 3, "dim": 6, "vdim": 5, "decay": [0.5, 0.9, 0.99], "rot": {"base": 100.0, "dims": 4}}
    moe = {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}}
    plain = {"kind": "moe", "expert": {"ff": 5}, "router": {"experts": 3, "top": 1}}
    return {"architecture": "Padulorn", "vocab": 30, "width": 24, "embedding": {"scale": 3.0}, "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_scale": 0.5,
            "layers": [{"type": "retention", "mixer": ret, "mlp": moe}, {"type": "attention", "mixer": att, "mlp": None},
                       {"type": "attention", "mixer": dict(att, v_mix=False, mask=None, rot=None), "mlp": plain},
                       {"type": "attention", "mixer": dict(att, heads=6), "mlp": moe}]}


def model_of(cfg, w):
    from paligemma_multimodal_system_b200.modeling_padulorn import PadulornConfig, PadulornForCausalLM
    return PadulornForCausalLM(PadulornConfig(cfg)).load_weights(w)


def test_config_rejects_what_the_design_does_not_have():
    from paligemma_multimodal_system_b200.modeling_padulorn import PadulornConfig, PadulornForCausalLM
    PadulornForCausalLM(PadulornConfig(cfg_small()))

    def broken(change):
        c = cfg_small()
        change(c["layers"])
        return PadulornForCausalLM(PadulornConfig(c))

    with pytest.raises(ValueError, match="unknown mixer type"):
        broken(lambda ls: ls[0].update(type="mlstm"))
    with pytest.raises(ValueError, match="feed-forward kind"):
        broken(lambda ls: ls[0]["mlp"].update(kind="dense"))
    with pytest.raises(ValueError, match="multiple of key/value heads"):
        broken(lambda ls: ls[2]["mixer"].update(kv_heads=3))
    with pytest.raises(ValueError, match="rotary"):
        broken(lambda ls: ls[1]["mixer"]["rot"].update(dims=12))
    with pytest.raises(ValueError, match="rotary"):
        broken(lambda ls: ls[0]["mixer"]["rot"].update(dims=3))
    with pytest.raises(ValueError, match="one decay per head"):
        broken(lambda ls: ls[0]["mixer"].update(decay=[0.5, 0.9]))
    with pytest.raises(ValueError, match="window"):
        broken(lambda ls: ls[1]["mixer"].update(mask={"size": 0}))
    with pytest.raises(ValueError, match="equal groups"):
        broken(lambda ls: ls[0]["mlp"]["router"].update(experts=7))
    with pytest.raises(ValueError, match="eligible"):
        broken(lambda ls: ls[0]["mlp"]["router"].update(top=5))
    with pytest.raises(ValueError, match="blends in"):
        broken(lambda ls: ls[3].update(mixer=dict(ls[3]["mixer"], vdim=7)))
    bad = cfg_small()
    bad["architecture"] = "Fadosun"
    with pytest.raises(ValueError):
        PadulornConfig(bad)


def test_every_tensor_is_accounted_for_and_the_cache_layout_follows_the_layers():
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=0)
    m = model_of(cfg, w)
    assert m.cache_layout() == [("state", (3, 6, 5)), ("kv", 20, 12), ("kv", 20, 12), ("kv", 20, 12)]
    assert [b.mixer.value_blend for b in m.blocks[1:]] == ["first", None, "later"] and m.blocks[1].ff is None
    assert (m.blocks[1].mixer.window, m.blocks[1].mixer.keep_first, m.blocks[2].mixer.window) == (7, 3, None)
    assert abs(m.blocks[1].mixer.rot_gain - (0.1 * math.log(4.0) + 1.0)) < 1e-12 and m.blocks[2].mixer.rot_gain == 1.0
    missing = dict(w)
    del missing["l3.mix.vmix"]
    with pytest.raises(KeyError, match="lacks l3.mix.vmix"):
        model_of(cfg, missing)
    # unused: no feed-forward there, no blending there
    model_of(cfg, dict(w, **{"l1.norm2": torch.zeros(24), "l2.mix.vmix": torch.zeros(())}))
    with pytest.raises(KeyError, match="without a place"):
        model_of(cfg, dict(w, **{"l0.mlp.e6.up": torch.zeros(9, 24)}))
    with pytest.raises(ValueError, match="l1.mix.q.norm"):
        model_of(cfg, dict(w, **{"l1.mix.q.norm": torch.zeros(10)}))  # one norm over the whole projection, not per head
    with pytest.raises(ValueError, match="l0.mix.g"):
        model_of(cfg, dict(w, **{"l0.mix.g": torch.zeros(3, 24)}))


def test_registry_picks_the_class_by_config(tmp_path):
    from paligemma_multimodal_system_b200 import registry
    assert "padulorn" in registry.known_architectures()
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=1)
    meta, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        meta[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(meta).encode()
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    m = registry.load_model(str(tmp_path), dtype=torch.float32)
    assert type(m).__name__ == "PadulornForCausalLM" and m.vocab_size == 30 and m.prec.f32
    assert float(m.blocks[3].mixer.w["vmix"]) == float(w["l3.mix.vmix"])


def test_a_step_scope_starts_empty_and_leaves_the_batch_alone():
    from paligemma_multimodal_system_b200.seq_ops import StepBatch, step_scope
    z = torch.zeros(1, dtype=torch.int32)
    b = StepBatch(T=1, E=1, max_n=1, tokens=z, pos=z, row_entry=z, row0=z, n=z, ctx=z, slot=z, page_table=z.view(1, 1), max_pages=1)
    s = step_scope(b)
    s.shared["values"] = 1
    assert b.shared is None and step_scope(s).shared == {} and s.tokens is b.tokens


def test_frequencies_of_product_and_oracle_agree_on_every_branch():
    from paligemma_multimodal_system_b200.mixers import ramped_rotary_frequencies, rotary_frequencies
    for rot in ({"base": 1e4, "dims": 32}, {"base": 1e4, "dims": 64, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                {"base": 30.0, "dims": 6, "scaling": {"factor": 2.0, "original": 20, "fast": 3.0, "slow": 3.0}},   # the ramp is a step
                {"base": 50.0, "dims": 8, "scaling": {"factor": 1.0, "original": 100, "fast": 4.0, "slow": 0.01}},  # gain one, end beyond the pairs
                {"base": 500.0, "dims": 8, "scaling": {"factor": 3.0, "original": 5, "fast": 9.0, "slow": 2.0}}):   # start clipped at zero
        f, gain = O.frequencies(rot)
        if rot.get("scaling"):
            got, g2 = ramped_rotary_frequencies(rot["base"], rot["dims"], *(rot["scaling"][k] for k in ("factor", "original", "fast", "slow")))
        else:
            got, g2 = rotary_frequencies(rot["base"], rot["dims"]), 1.0
        assert torch.allclose(got, torch.tensor(f, dtype=torch.float64), rtol=1e-12) and abs(g2 - gain) < 1e-12


def test_oracle_retention_equals_its_unrolled_sum():
    g = torch.Generator().manual_seed(1)
    T, H, dim, vdim = 9, 2, 4, 3
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (dim, dim, vdim))
    a = torch.tensor([0.3, 1.0], dtype=torch.float64)
    o = O.retained(q, k, v, a)
    for h in range(H):
        for t in range(T):
            assert torch.allclose(o[t, h], sum(float(a[h]) ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1)))


def test_oracle_rotations_depend_on_the_distance_only_and_leave_the_rest():
    v, u = torch.randn(10, dtype=torch.float64), torch.randn(10, dtype=torch.float64)
    for partner in ("next", "half"):
        rot = {"base": 50.0, "dims": 6}
        t = O.turned(v, 7, rot, partner)
        assert torch.equal(t[6:], v[6:]) and torch.equal(O.turned(v, 0, rot, partner), v) and torch.allclose(t.norm(), v.norm())
        assert torch.allclose(O.turned(u, 11, rot, partner) @ t, O.turned(u, 5, rot, partner) @ O.turned(v, 1, rot, partner))
        gained = O.turned(v, 7, dict(rot, scaling={"factor": 2.0, "original": 1e9, "fast": 2.0, "slow": 1.0}), partner)
        assert abs(float(gained[:6].norm() / v[:6].norm()) - (1.0 + 0.1 * math.log(2.0))) < 1e-12
    assert O.turned(v, 3, None, "half") is v


def test_oracle_mask_edges():
    mask = {"size": 4, "keep_first": 2}
    assert [j for j in range(12) if O.visible(9, j, mask)] == [0, 1, 6, 7, 8, 9]
    assert [j for j in range(12) if O.visible(1, j, mask)] == [0, 1] and [j for j in range(5) if O.visible(3, j, None)] == [0, 1, 2, 3]


def test_oracle_choice_of_experts():
    z = torch.tensor([3.0, -4.0, -4.0, 1.0, 1.2, -5.0, 0.9, 0.8, -5.0])  # best single in group 0, best pair in group 1
    pick = O.chosen(z, {"experts": 9, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert [e for e, _ in pick] == [4, 3] and torch.allclose(torch.stack([w for _, w in pick]), torch.sigmoid(z[[4, 3]]))
    assert [e for e, _ in O.chosen(z, {"experts": 9, "top": 3, "groups": {"count": 3, "keep": 2}})] == [4, 3, 6]
    assert [e for e, _ in O.chosen(z, {"experts": 9, "top": 2})] == [0, 4]


def test_oracle_blends_values_from_the_first_blending_layer():
    cfg = cfg_small()
    w = {k: v.double() for k, v in O.random_weights(cfg, seed=2).items()}
    x = torch.randn(5, 24, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    m = cfg["layers"][3]["mixer"]
    alone, own = O.attention(x, w, "l3.mix.", m, 1e-5)
    assert torch.allclose(O.attention(x, w, "l3.mix.", m, 1e-5, own)[0], alone)  # blending its own values changes nothing
    zero = O.attention(x, w, "l3.mix.", m, 1e-5, torch.zeros_like(own))[0]
    assert torch.allclose(zero, (1.0 - w["l3.mix.vmix"]) * alone)


def test_oracle_whole_equals_prefix():
    """Causality of the restatement itself: logits of a prefix do not change when tokens follow."""
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=4)
    tk = torch.randint(0, 30, (20,), generator=torch.Generator().manual_seed(5)).tolist()
    a, b = O.forward(cfg, w, tk), O.forward(cfg, w, tk[:11])
    assert torch.allclose(a[:11], b, atol=1e-9)
