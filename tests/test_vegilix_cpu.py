"""Host side of the Vegilix design, no GPU: registry and configuration reading, the layer loop, checkpoint packing, and the
float64 oracle's own consistency (portions == whole, mask, wavelength scaling, difference of maps, retention, routing)."""
import copy
import math
import os

import pytest
import torch

from tests import vegilix_plain as P
from tests import vegilix_util as U

LAYERS = [U.attention(mlp=U.moe()), U.retention(mlp=U.moe(experts=5, top=1, ff=12, shared_ff=0)),
          U.attention(heads=4, kv_heads=4, dim=8, vdim=5, window=40, keep=0, dims=8, scaling=None, diff=0.2),
          U.retention(heads=2, dim=6, vdim=9, dims=0, decay=[0.5, 0.97])]


def _ckpt(tmp_path, layers, seed=0, **kw):
    cfg = U.config(layers, **kw)
    tensors = U.random_tensors(cfg, seed)
    return cfg, tensors, U.write_checkpoint(str(tmp_path / "ckpt"), cfg, tensors)


def test_registry_and_spec(tmp_path):
    from ssd_b200 import lib as L
    from ssd_b200.config import load_hf_config
    from ssd_b200.hybrid import HybridSpec
    _, _, path = _ckpt(tmp_path, LAYERS, width=24, vocab=31, eps=1e-4, loop=(1, 3, 2), mult=0.7)
    hf = load_hf_config(path)
    assert hf.family.name == "vegilix" and hf.family.kind == "hybrid" and hf.vocab_size == 31
    s = HybridSpec.from_dir(path)
    assert (s.width, s.vocab, s.eps, s.residual_mult, s.loop) == (24, 31, 1e-4, 0.7, (1, 3, 2))
    assert s.block == L.BLOCK_SERIAL_SANDWICH and s.norm_offset == 1.0 and not s.tied_head and s.has_cache and s.has_state
    a, b, c, d = s.layers
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.attn_scale, a.maps, a.diff) == ("attention", 6, 2, 10, 14, 24, 3, 0.4, 2, 0.4)
    assert (a.rot_dims, a.rot_base, a.rot_half, a.qk_norm, a.learned_sink, a.conv) == (6, 300.0, 1, 3, 0, 1)
    assert (a.wave_factor, a.wave_low, a.wave_high, a.wave_original) == (3.0, 0.8, 2.5, 60.0)
    assert (a.mlp, a.experts, a.top, a.ff, a.shared_ff, a.route_top_softmax, a.expert_glu, a.expert_act, a.shared_gate) == ("moe", 6, 2, 20, 12, 1, 1, L.ACT_SILU, 0)
    assert (b.mixer, b.heads, b.dim, b.vdim, b.rot_dims, b.rot_base, b.decay) == ("retention", 3, 12, 7, 8, 500.0, (0.75, 0.9375, 0.984375))
    assert (b.top, b.shared_ff, c.mlp, c.keep_first, c.wave_factor, d.rot_dims, d.decay) == (1, 0, None, 0, 0.0, 0, (0.5, 0.97))
    assert s.runs == [0, 1, 2, 1, 2, 3]
    c_cfg = a.cfg()
    assert (c_cfg.maps, c_cfg.keep_first, c_cfg.window) == (2, 3, 24) and abs(c_cfg.diff - 0.4) < 1e-6


def test_layer_loop():
    from ssd_b200.hybrid import HybridSpec
    layers = [U.retention() for _ in range(4)]
    for loop, want in ((None, [0, 1, 2, 3]), ((0, 4, 2), [0, 1, 2, 3] * 2), ((2, 3, 3), [0, 1, 2, 2, 2, 3]), ((1, 3, 1), [0, 1, 2, 3]), ((3, 4, 2), [0, 1, 2, 3, 3])):
        cfg = U.config(layers, loop=loop)
        assert HybridSpec.from_config(cfg).runs == want == P.layer_runs(cfg)
    for loop in ((1, 1, 2), (2, 5, 2), (0, 2, 0), (-1, 2, 2)):
        with pytest.raises(ValueError):
            HybridSpec.from_config(U.config(layers, loop=loop))
    bad = U.config([U.retention(heads=3, decay=[0.5, 0.5])])
    with pytest.raises(ValueError):
        HybridSpec.from_config(bad)
    with pytest.raises(ValueError):
        HybridSpec.from_config(U.config([{"type": "wkv", "mixer": {"heads": 1, "dim": 4}, "mlp": None}]))


def test_packing_matches_the_bound_layout(tmp_path):
    from ssd_b200.hybrid import HybridSpec, pack_hybrid_weights, read_safetensors
    cfg, tensors, path = _ckpt(tmp_path, LAYERS, loop=(0, 2, 3))
    raw = read_safetensors(os.path.join(path, "model.safetensors"))
    assert set(raw) == set(tensors)
    w = pack_hybrid_weights(HybridSpec.from_dir(path), raw, torch.float32, "cpu")
    assert len(w["layers"]) == 4        # a looped layer is packed once
    assert w["HEAD"] is not w["EMBED"] and torch.equal(w["HEAD"], tensors["head"])
    l0, l1, l2, l3 = w["layers"]
    assert l0["ATTN_IN"].shape == (2 * 6 * 10 + 2 * 2 * 10 + 2 * 14, 40) and torch.equal(l0["ATTN_IN"][120:160], tensors["l0.mix.k"])
    assert torch.equal(l0["ATTN_QK_NORM"], torch.stack([tensors["l0.mix.q.norm"], tensors["l0.mix.k.norm"]]))
    assert torch.equal(l0["ATTN_DIFF"], torch.stack([tensors["l0.mix." + s] for s in ("lq1", "lk1", "lq2", "lk2")]))
    assert torch.equal(l0["NORM_POST"], tensors["l0.norm1b"]) and torch.equal(l0["NORM2"], tensors["l0.norm2"]) and torch.equal(l0["NORM2_POST"], tensors["l0.norm2b"])
    assert l0["EXPERT_IN"].shape == (6, 40, 40) and torch.equal(l0["EXPERT_IN"][4][:20], tensors["l0.mlp.e4.gate"]) and torch.equal(l0["EXPERT_IN"][4][20:], tensors["l0.mlp.e4.up"])
    assert l0["SHARED_IN"].shape == (24, 40) and "SHARED_IN" not in l1 and "CONV_W" not in l0 and "LS_MIX" not in l0 and "ATTN_SINK" not in l0
    assert l1["RET_IN"].shape == (2 * 3 * 12 + 2 * 3 * 7, 40) and torch.equal(l1["RET_IN"][72 + 21:], tensors["l1.mix.g"])
    assert "NORM2" not in l2 and "NORM2_POST" not in l3 and torch.equal(l3["MIX_OUT"], tensors["l3.mix.o"])


def test_oracle_portions_equal_whole(tmp_path):
    cfg, tensors, _ = _ckpt(tmp_path, LAYERS, loop=(1, 3, 2))
    m = P.PlainModel(cfg, tensors)
    toks = torch.randint(0, 50, (60,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = m.run(toks)
    st, out, pos = m.new_state(), [], 0
    assert len(st) == 6
    for c in (7, 2, 1, 13, 7, 30):
        out.append(m.run(toks[pos:pos + c], st, pos))
        pos += c
    assert torch.allclose(torch.cat(out), whole, rtol=1e-10, atol=1e-10)


def test_oracle_mask():
    mask = {"size": 4, "keep_first": 2}

    def seen(i, m=mask):
        return [j for j in range(12) if bool(P.visible(torch.tensor(i), torch.tensor(j), m))]
    assert seen(0) == [0] and seen(1) == [0, 1] and seen(3) == [0, 1, 2, 3]
    assert seen(5) == [0, 1, 2, 3, 4, 5] and seen(6) == [0, 1, 3, 4, 5, 6] and seen(9) == [0, 1, 6, 7, 8, 9]
    assert seen(9, {"size": 4, "keep_first": 0}) == [6, 7, 8, 9] and seen(9, None) == list(range(10)) and seen(5, {"size": 1, "keep_first": 4}) == [0, 1, 2, 3, 5]
    # a window of one without kept keys returns the value rows themselves
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(9, 5, generator=g, dtype=P.F64) for _ in range(3))
    assert torch.allclose(P.masked_softmax_attention(q, k, v, 0, 0.7, {"size": 1, "keep_first": 0}), v)


def test_oracle_rotation():
    rot = {"base": 300.0, "dims": 6, "scaling": U.SCALING}
    plain = [300.0 ** (-2 * i / 6) for i in range(3)]
    f = P.rotary_frequencies(rot)
    waves = [2 * math.pi / x for x in plain]
    sc = U.SCALING
    assert waves[0] < sc["original"] / sc["high"] < waves[1] < sc["original"] / sc["low"] < waves[2]   # one frequency of each kind
    assert f[0] == plain[0] and abs(f[2] - plain[2] / 3.0) < 1e-15 and plain[1] / 3.0 < f[1] < plain[1]
    assert P.rotary_frequencies({"base": 300.0, "dims": 6}) == plain
    # entry i turns with entry i + dims/2, lengths stay, products of rotated vectors depend on the distance only
    a, b = torch.randn(1, 1, 10, dtype=P.F64), torch.randn(1, 1, 10, dtype=P.F64)
    ra, rb = P.rotate_half(a, 17, rot), P.rotate_half(b, 12, rot)
    assert torch.equal(ra[..., 6:], a[..., 6:]) and abs(float(ra[0, 0, [0, 3]].norm() - a[0, 0, [0, 3]].norm())) < 1e-12
    assert abs(float((ra * rb).sum() - (P.rotate_half(a, 105, rot) * P.rotate_half(b, 100, rot)).sum())) < 1e-9


def test_oracle_difference_and_retention():
    z = torch.zeros(4, dtype=P.F64)
    assert float(P.difference_weight(z, z, z, z, 0.3)) == 0.3
    o = torch.ones(4, dtype=P.F64)
    assert abs(float(P.difference_weight(o, o / 4, z, z, 0.0)) - (math.e - 1.0)) < 1e-12
    a1, a2 = torch.randn(3, 8, dtype=P.F64), torch.randn(3, 8, dtype=P.F64)
    y = P.difference_heads(a1, a2, 0.5, 0.25, 0.0)
    assert torch.allclose((y ** 2).mean(-1), torch.full((3,), 0.75 ** 2, dtype=P.F64)) and torch.allclose(P.difference_heads(2 * a1, 2 * a2, 0.5, 0.25, 0.0), y)
    # the recurrence equals the sum over the past, o_t = sum_j a^(t - j) (q_t . k_j) v_j
    q, k, v = torch.randn(7, 5, dtype=P.F64), torch.randn(7, 5, dtype=P.F64), torch.randn(7, 3, dtype=P.F64)
    S, a = torch.zeros(5, 3, dtype=P.F64), 0.8
    for t in range(7):
        S, o = P.retention_step(S, q[t], k[t], v[t], a)
        assert torch.allclose(o, sum(a ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)))


def test_oracle_routing_and_norms():
    z = torch.tensor([0.5, 2.0, -1.0, 2.0, 1.0], dtype=P.F64)
    chosen, w = P.route_top(z, 3)
    assert chosen == [1, 3, 4] and abs(float(w.sum()) - 1.0) < 1e-12 and abs(float(w[0] / w[2]) - math.e) < 1e-9   # ties to the lower index
    assert P.route_top(z, 1)[1].tolist() == [1.0]
    x = torch.randn(2, 6, dtype=P.F64)
    assert torch.equal(P.rms_norm_offset(x, torch.zeros(6, dtype=P.F64), 1e-5), P.unit_rms(x, 1e-5))


def test_every_constant_of_the_configuration_matters():
    """Each number of config.json moves the oracle: a reader that drops one cannot pass the comparisons of the GPU tests."""
    cfg = U.config([U.attention(mlp=U.moe()), U.retention(mlp=U.moe())], loop=(0, 1, 2))
    tensors = U.random_tensors(cfg, 1)
    toks = torch.randint(0, 50, (70,), generator=torch.Generator().manual_seed(2)).tolist()
    ref = P.PlainModel(cfg, tensors).run(toks)
    a, r = ("layers", 0, "mixer"), ("layers", 1, "mixer")
    for path, val in ((a + ("scale",), 0.5), (a + ("diff",), 0.5), (a + ("mask", "size"), 23), (a + ("mask", "keep_first"), 4), (a + ("rot", "base"), 350.0),
                      (a + ("rot", "dims"), 4), (a + ("rot", "scaling", "factor"), 4.0), (a + ("rot", "scaling", "low"), 0.6),
                      (a + ("rot", "scaling", "high"), 3.0), (a + ("rot", "scaling", "original"), 80), (r + ("rot", "base"), 600.0), (r + ("rot", "dims"), 6),
                      (r + ("decay", 1), 0.9), (("layers", 0, "mlp", "router", "top"), 3), (("norm", "eps"), 1e-2), (("residual_mult",), 0.5),
                      (("loop", "times"), 3), (("loop", "stop"), 2)):
        other = copy.deepcopy(cfg)
        node = other
        for key in path[:-1]:
            node = node[key]
        assert node[path[-1]] != val
        node[path[-1]] = val
        assert U.rel_err(P.PlainModel(other, tensors).run(toks).numpy(), ref.numpy()) > 3e-3, path
