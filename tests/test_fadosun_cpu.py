"""Host-side parts of the Fadosun decoder (configuration, weight accounting, cache layout, registry, channel layouts) and the oracle against
itself; no GPU."""
import json
import math
import os
import struct
import sys

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from oracle import fadosun_oracle as O  # noqa: E402


def cfg_small():
    delta = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "conv": 3}
    left = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3, "rot": {"base": 100.0, "dims": 4}}
    right = {"heads": 3, "groups": 1, "state": 5, "vdim": 4, "conv": 4, "norm_groups": 2}
    mem = {"heads": 2, "dim": 7, "vdim": 9, "gate_cap": 5.0}
    return {"architecture": "Fadosun", "vocab": 30, "width": 24, "norm": {"eps": 1e-5}, "layers": [
        {"type": "channel_delta", "mixer": delta, "mlp": {"kind": "dense", "ff": 20}},
        {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.7, "right_scale": 1.4}, "mlp": None},
        {"type": "mlstm", "mixer": mem, "mlp": {"kind": "dense", "ff": 9}}]}


def model_of(cfg, w):
    from paligemma_multimodal_system_b200.modeling_fadosun import FadosunConfig, FadosunForCausalLM
    return FadosunForCausalLM(FadosunConfig(cfg)).load_weights(w)


def test_config_rejects_what_the_design_does_not_have():
    from paligemma_multimodal_system_b200.modeling_fadosun import FadosunConfig, FadosunForCausalLM
    FadosunForCausalLM(FadosunConfig(cfg_small()))

    def broken(change, where=FadosunForCausalLM):
        c = cfg_small()
        change(c["layers"])
        return where(FadosunConfig(c)) if where is FadosunForCausalLM else FadosunConfig(c)

    with pytest.raises(ValueError, match="unknown mixer type"):
        broken(lambda ls: ls[0].update(type="attention"))
    with pytest.raises(ValueError, match="feed-forward kind"):
        broken(lambda ls: ls[0]["mlp"].update(kind="moe"))
    with pytest.raises(ValueError, match="multiple of query/key heads"):
        broken(lambda ls: ls[0]["mixer"].update(kv_heads=3))
    with pytest.raises(ValueError, match="taps"):
        broken(lambda ls: ls[0]["mixer"].update(conv=9))
    with pytest.raises(ValueError, match="multiple of key/value heads"):
        broken(lambda ls: ls[1]["mixer"]["left"].update(kv_heads=3))
    with pytest.raises(ValueError, match="rotary"):
        broken(lambda ls: ls[1]["mixer"]["left"]["rot"].update(dims=5))
    with pytest.raises(ValueError, match="B / C groups"):
        broken(lambda ls: ls[1]["mixer"]["right"].update(groups=2))
    with pytest.raises(ValueError, match="norm's groups"):
        broken(lambda ls: ls[1]["mixer"]["right"].update(norm_groups=5))
    with pytest.raises(ValueError, match="cap"):
        broken(lambda ls: ls[2]["mixer"].update(gate_cap=0.0))
    bad = cfg_small()
    bad["architecture"] = "Mapedra"
    with pytest.raises(ValueError):
        FadosunConfig(bad)


def test_every_tensor_is_accounted_for_and_the_cache_layout_follows_the_layers():
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=0, rank=(3, 11))
    m = model_of(cfg, w)
    # delta: state, convolution inputs (q and k channels padded to multiples of 8: 16 + 16 + 24); parallel: pages, state, convolution
    # inputs (16 + 8 + 8); matrix memory: state, normaliser + maximum once per block of value columns (9 columns: blocks of 16)
    assert m.cache_layout() == [("state", (4, 6, 5)), ("state", (2, 56)), ("kv", 16, 12), ("state", (3, 5, 4)), ("state", (3, 32)), ("state", (2, 7, 9)), ("state", (1, 2, 8))]
    assert m.cache_at == [0, 2, 5] and m.blocks[1].ff is None and m.blocks[1].sub2 is None
    assert m.blocks[1].mixer.left.out_scale == 0.7 and m.blocks[1].mixer.right.out_scale == 1.4
    assert m.blocks[0].mixer.w["a1"].shape == (3, 24) and m.blocks[0].mixer.w["g1"].shape == (11, 24)  # ranks come from the checkpoint
    missing = dict(w)
    del missing["l2.mix.i.b"]
    with pytest.raises(KeyError, match="lacks l2.mix.i.b"):
        model_of(cfg, missing)
    model_of(cfg, dict(w, **{"l1.norm2": torch.zeros(24)}))  # unused: the layer has no feed-forward
    extra = dict(w, **{"l1.mlp.up": torch.zeros(20, 24)})
    with pytest.raises(KeyError, match="without a place"):
        model_of(cfg, extra)
    with pytest.raises(ValueError, match="l0.mix.a2"):
        model_of(cfg, dict(w, **{"l0.mix.a2": torch.zeros(24, 4)}))  # does not fit a1's rank
    with pytest.raises(ValueError, match="l1.mix.right.in"):
        model_of(cfg, dict(w, **{"l1.mix.right.in": torch.zeros(30, 24)}))
    one_tap = cfg_small()
    one_tap["layers"][0]["mixer"]["conv"] = 1
    assert model_of(one_tap, O.random_weights(one_tap, seed=0)).cache_layout()[1] is None  # nothing to remember


def test_registry_picks_the_class_by_config(tmp_path):
    from paligemma_multimodal_system_b200 import registry
    assert "fadosun" in registry.known_architectures()
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
    assert type(m).__name__ == "FadosunForCausalLM" and m.vocab_size == 30 and m.prec.f32
    assert torch.equal(m.blocks[0].mixer.w["A_log"].float(), w["l0.mix.A_log"])


def test_state_slots_and_pages_of_a_mixed_layout():
    """One store holds pages and several state tensors per layer; a released request's slot and pages are the next one's."""
    from paligemma_multimodal_system_b200.cache import SequenceStore
    m = model_of(cfg_small(), O.random_weights(cfg_small(), seed=0))
    st = SequenceStore(m.cache_layout(), max_tokens=128, num_slots=2, dtype=torch.float32, device="cpu")
    assert [None if s is None else tuple(s.shape) for s in st.state] == [(2, 4, 6, 5), (2, 2, 56), None, (2, 3, 5, 4), (2, 3, 32), (2, 2, 7, 9), (2, 1, 2, 8)]
    assert all(s is None or s.dtype == torch.float32 for s in st.state) and st.k_pages[2].shape == (2, 64, 16) and st.v_pages[2].shape == (2, 64, 12)
    st.admit("a"), st.admit("b")
    assert st.reserve("a", 64).pages == [0] and st.reserve("b", 3).pages == [1] and (st.live["a"].slot, st.live["b"].slot) == (0, 1)
    st.release("a")
    st.admit("c")
    assert st.reserve("c", 10).pages == [0] and st.live["c"].slot == 0


def test_oracle_delta_rule_against_its_definition():
    """With unit decay and beta = 1, writing an orthonormal set of keys makes S^T k_j = v_j exactly; a second write along a key replaces."""
    H, dim, vdim = 1, 5, 3
    k = torch.eye(dim, dtype=torch.float64)[:, None]
    v = torch.randn(dim, H, vdim, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    q = k[[4, 3, 2, 1, 0]]
    ones = torch.ones(dim, H, dtype=torch.float64)
    o = O.delta_rule(torch.cat([q, k[:1]]), torch.cat([k, k[:1]]), torch.cat([v, -v[:1]]), torch.cat([ones, ones[:1]]), torch.ones(dim + 1, H, dim, dtype=torch.float64))
    assert torch.allclose(o[4], v[0]) and torch.allclose(o[5], -v[0]) and torch.allclose(o[0], torch.zeros(H, vdim, dtype=torch.float64))
    # the decay acts on the key's row before the write
    g = torch.ones(2, H, dim, dtype=torch.float64)
    g[1, 0, 0] = 0.25
    o = O.delta_rule(k[[1, 0]], k[:2], v[:2], ones[:2], g)
    assert torch.allclose(o[1], 0.25 * v[0])


def test_oracle_state_space_equals_its_unrolled_sum():
    g = torch.Generator().manual_seed(1)
    T, H, N, vdim = 9, 2, 4, 3
    x, B, C = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (vdim, N, N))
    dt, r = torch.rand(T, H, generator=g, dtype=torch.float64), torch.tensor([0.5, 2.0], dtype=torch.float64)
    y = O.state_space(x, B, C, dt, r)
    for h in range(H):
        for t in range(T):
            want = sum(math.exp(-float(r[h] * dt[j + 1:t + 1, h].sum())) * dt[j, h] * (C[t, h] @ B[j, h]) * x[j, h] for j in range(t + 1))
            assert torch.allclose(y[t, h], want)


def test_oracle_matrix_memory_equals_the_form_without_a_running_maximum():
    """The stabiliser cancels except in the floor of the denominator: o = S~^T q / (max(|n~ . q|, 1) + 1e-6 e^m) with raw exponentials."""
    g = torch.Generator().manual_seed(2)
    T, H, dim, vdim = 12, 2, 5, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (dim, dim, vdim))
    i, f = 2.0 * torch.randn(T, H, generator=g, dtype=torch.float64), -torch.rand(T, H, generator=g, dtype=torch.float64)
    o = O.matrix_memory(q, k, v, i, f)
    for h in range(H):
        S, n, m = torch.zeros(dim, vdim, dtype=torch.float64), torch.zeros(dim, dtype=torch.float64), 0.0
        for t in range(T):
            S = math.exp(f[t, h]) * S + math.exp(i[t, h]) * torch.outer(k[t, h], v[t, h])
            n = math.exp(f[t, h]) * n + math.exp(i[t, h]) * k[t, h]
            m = max(float(f[t, h]) + m, float(i[t, h]))
            want = S.T @ q[t, h] / (max(abs(float(n @ q[t, h])), 1.0) + 1e-6 * math.exp(m))
            assert torch.allclose(o[t, h], want)


def test_oracle_convolution_rotation_and_norms():
    u = torch.arange(12.0).reshape(4, 3)
    w = torch.zeros(3, 3)
    w[:, 2] = 1.0  # the last tap is the token itself
    assert torch.equal(O.short_conv(u, w), u)
    w = torch.zeros(3, 3)
    w[:, 0] = 1.0  # the first tap is two tokens back; nothing before the start
    assert torch.equal(O.short_conv(u, w, torch.ones(3)), torch.cat([torch.zeros(2, 3), u[:2]]) + 1.0)
    v = torch.randn(5, 10, dtype=torch.float64)
    t = O.turn_half(v, 7, 50.0, 6)
    assert torch.equal(t[:, 6:], v[:, 6:]) and torch.allclose(t[:, 0] ** 2 + t[:, 3] ** 2, v[:, 0] ** 2 + v[:, 3] ** 2) and torch.equal(O.turn_half(v, 0, 50.0, 6), v)
    x = torch.randn(4, 32, dtype=torch.float64)
    y = O.layer_norm(x, torch.ones(32, dtype=torch.float64), torch.zeros(32, dtype=torch.float64), 0.0)
    assert torch.allclose(y.mean(-1), torch.zeros(4, dtype=torch.float64), atol=1e-12) and torch.allclose((y * y).mean(-1), torch.ones(4, dtype=torch.float64))


def test_oracle_logistic_attention_is_not_normalised():
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=3)
    h = torch.randn(6, 24, generator=torch.Generator().manual_seed(2))
    m = dict(cfg["layers"][1]["mixer"]["left"], scale=0.0)  # every weight is sigmoid(bias of the head)
    v = (h @ w["l1.mix.left.v"].T).view(6, 2, 6).cumsum(0)[:, [0, 0, 1, 1]]
    want = (v * torch.sigmoid(w["l1.mix.left.pb"])[:, None]).reshape(6, -1) @ w["l1.mix.left.o"].T
    assert torch.allclose(O.logistic_attention(h, w, "l1.mix.left.", m), want, atol=1e-5)


def test_oracle_whole_equals_prefix():
    """Causality of the restatement itself: logits of a prefix do not change when tokens follow."""
    cfg = cfg_small()
    w = O.random_weights(cfg, seed=4)
    tk = torch.randint(0, 30, (20,), generator=torch.Generator().manual_seed(5)).tolist()
    a, b = O.forward(cfg, w, tk), O.forward(cfg, w, tk[:11])
    assert torch.allclose(a[:11], b, atol=1e-9)


def test_library_and_host_agree_on_the_normaliser_blocks():
    from paligemma_multimodal_system_b200 import _lib, build, seq_ops
    build.build()
    for v in (1, 4, 7, 16, 24, 64, 128, 130):
        assert _lib.lib().pg_recurrence_block(v) == seq_ops.recurrence_block(v)
