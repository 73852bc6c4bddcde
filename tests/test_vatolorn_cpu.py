"""Host side of the Vatolorn design, no GPU: registry and configuration reading, checkpoint packing, and the float64
oracle's own consistency (portions == whole, chunk edges, streams, delta rule, rotation, norms)."""
import math
import os

import pytest
import torch

from tests import vatolorn_plain as P
from tests import vatolorn_util as U


def _ckpt(tmp_path, layers, seed=0, **kw):
    cfg = U.config(layers, **kw)
    tensors = U.random_tensors(cfg, seed)
    return cfg, tensors, U.write(str(tmp_path / "ckpt"), cfg, tensors)


LAYERS = [U.parallel(mlp=U.dense()),
          U.parallel(U.attention(heads=4, kv_heads=4, dim=8, vdim=12, conv=1, chunk=40, scale=0.5, dims=8, scaling=None),
                     U.delta(heads=2, kv_heads=2, dim=5, vdim=9, conv=1, decay_rank=8, gate_rank=1)),
          U.parallel(U.attention(heads=5, kv_heads=1, dim=6, vdim=3, conv=3, chunk=7, dims=0),
                     U.delta(heads=4, kv_heads=1, dim=20, vdim=3, conv=5, decay_rank=17, gate_rank=4), mlp=U.dense(ff=33))]


def test_registry_and_spec(tmp_path):
    from ssd_b200 import lib as L
    from ssd_b200.config import load_hf_config
    from ssd_b200.hybrid import HybridSpec
    _, _, path = _ckpt(tmp_path, LAYERS, width=24, vocab=31, eps=1e-4, streams=5, logit_scale=1.5)
    hf = load_hf_config(path)
    assert hf.family.name == "vatolorn" and hf.family.kind == "hybrid" and hf.vocab_size == 31
    s = HybridSpec.from_dir(path)
    assert (s.width, s.vocab, s.eps, s.streams, s.logit_scale, len(s.layers)) == (24, 31, 1e-4, 5, 1.5, 3)
    assert s.block == L.BLOCK_SERIAL_PRENORM and s.norm_offset == 0.0 and not s.tied_head and not s.gated_residual
    assert s.has_cache and s.has_state
    a, b, c = s.layers
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.pair_conv, a.chunk, a.window, a.attn_scale) == ("parallel", 6, 2, 10, 6, 4, 24, 0, 0.4)
    assert (a.rot_dims, a.rot_base, a.yarn_factor, a.yarn_original, a.yarn_fast, a.yarn_slow, a.rot_half) == (6, 300.0, 3.0, 80.0, 6.0, 0.5, 0)
    assert (a.qk_norm, a.sink, a.pair_gate, a.pair_norm, a.left_scale, a.right_scale) == (2, 0.0, 0, 1, 0.5, 0.5)
    assert (a.d_heads, a.d_kv_heads, a.d_dim, a.d_vdim, a.conv, a.d_decay_rank, a.d_gate_rank, a.d_gate_act) == (6, 3, 12, 7, 3, 5, 9, 1)
    assert (a.mlp, a.ff, a.ff_act) == ("dense", 28, L.ACT_SILU) and b.mlp is None
    assert (b.yarn_factor, b.rot_dims, b.pair_conv, b.d_gate_rank) == (0.0, 8, 1, 1) and (c.rot_dims, c.chunk, c.d_decay_rank) == (0, 7, 17)
    assert (a.cfg().d_decay_rank, a.cfg().d_gate_rank, c.cfg().d_decay_rank) == (8, 16, 24)   # bound in whole vectors of 8
    with pytest.raises(ValueError):   # the ranks are not in the configuration
        HybridSpec.from_config(U.config(LAYERS))
    with pytest.raises(ValueError):
        HybridSpec.from_config(U.config([{"type": "rglru", "mixer": {"width": 4, "blocks": 1, "conv": 2}, "mlp": None}]))
    # the older pair keeps its own variant: gated heads, a sink, unit norms per head, one decay per head
    from tests import kefurax_util as K
    k = HybridSpec.from_config(K.config([K.parallel(mlp=K.dense())])).layers[0]
    assert (k.qk_norm, k.sink, k.pair_gate, k.pair_norm, k.d_decay_rank, k.d_gate_rank, k.d_gate_act, k.chunk, k.ff_act) == (1, 1.0, 1, 0, 0, 0, 0, 0, L.ACT_GELU_TANH)


def test_packing_matches_the_bound_layout(tmp_path):
    from ssd_b200.hybrid import HybridSpec, pack_hybrid_weights, read_safetensors
    _, t, path = _ckpt(tmp_path, LAYERS, streams=3)
    raw = read_safetensors(os.path.join(path, "model.safetensors"))
    assert set(raw) == set(t)
    w = pack_hybrid_weights(HybridSpec.from_dir(path), raw, torch.float32, "cpu")
    l0, l1, l2 = w["layers"]
    # attention q | k | v, delta q | k | v, beta, the two bottlenecks padded with zero rows to a multiple of 8
    rows = [60, 20, 12, 36, 36, 42, 6, 8, 16]
    o = [sum(rows[:i]) for i in range(len(rows) + 1)]
    assert l0["PAIR_IN"].shape == (o[-1], 40)
    for i, name in enumerate(["left.q", "left.k", "left.v", "right.q", "right.k", "right.v", "right.b", "right.a1", "right.g1"]):
        n = t["l0.mix." + name].shape[0]
        assert torch.equal(l0["PAIR_IN"][o[i]:o[i] + n], t["l0.mix." + name]) and not l0["PAIR_IN"][o[i] + n:o[i + 1]].any()
    assert l0["DELTA_A2"].shape == (72, 8) and torch.equal(l0["DELTA_A2"][:, :5], t["l0.mix.right.a2"]) and not l0["DELTA_A2"][:, 5:].any()
    assert l0["DELTA_G2"].shape == (42, 16) and torch.equal(l0["DELTA_G2"][:, :9], t["l0.mix.right.g2"])
    assert torch.equal(l0["ATTN_IN_B"][60:80], t["l0.mix.left.k.b"]) and torch.equal(l0["ATTN_CONV_W"][80:], t["l0.mix.left.v.conv"])
    assert torch.equal(l0["ATTN_QK_NORM"], torch.cat([t["l0.mix.left.q.norm"], t["l0.mix.left.k.norm"]]))
    assert l0["CONV_W"].shape == (114, 3) and torch.equal(l0["CONV_W"][36:72], t["l0.mix.right.k.conv"])
    assert torch.equal(l0["MIX_NORM"], t["l0.mix.right.norm"].repeat(6)) and l0["DELTA_DT_B"].shape == (72,)
    assert torch.equal(l0["PAIR_NORM"][0], t["l0.mix.left.out"]) and torch.equal(l0["PAIR_NORM"][1], t["l0.mix.right.out"])
    # stream coefficients: the mixer's first, the feed-forward's second; a layer without one has only the first
    assert l0["HC_MIX"].shape == (2, 3, 3) and torch.equal(l0["HC_MIX"][1], t["l0.hc2.mix"]) and torch.equal(l0["HC_IN"][0], t["l0.hc1.in"])
    assert l1["HC_MIX"].shape == (1, 3, 3) and l1["HC_OUT"].shape == (1, 3) and "NORM2" not in l1 and "GLU_IN" not in l1
    assert torch.equal(l2["GLU_IN"][33:], t["l2.mlp.up"]) and torch.equal(l2["NORM2"], t["l2.norm2"]) and "LS_MIX" not in l2
    assert l1["DELTA_G2"].shape == (18, 8) and l2["DELTA_A2"].shape == (80, 24)


def test_oracle_portions_equal_whole(tmp_path):
    cfg, tensors, _ = _ckpt(tmp_path, LAYERS, streams=4)
    m = P.PlainModel(cfg, tensors)
    toks = torch.randint(0, 50, (60,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = m.run(toks)
    st, out, pos = {}, [], 0
    for c in (7, 2, 1, 13, 7, 30):
        out.append(m.run(toks[pos:pos + c], state=st, p0=pos))
        pos += c
    assert torch.allclose(torch.cat(out), whole, rtol=1e-10, atol=1e-10)


def test_oracle_chunks_and_rotation():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(9, 5, generator=g, dtype=P.F64) for _ in range(3))
    assert [P.first_visible(i, 4) for i in (0, 3, 4, 7, 8, 11)] == [0, 0, 4, 4, 8, 8] and P.first_visible(10, 0) == 0
    # the first position of a chunk sees itself only; the last one sees the whole chunk and nothing before it
    o = P.chunked_softmax_attention(q, k, v, 0, 0.7, 4)
    assert torch.allclose(o[[0, 4, 8]], v[[0, 4, 8]])
    k2, v2 = k.clone(), v.clone()
    k2[3], v2[3] = 100.0 * q[4], 50.0       # a key that would dominate, one position before the chunk
    assert torch.allclose(P.chunked_softmax_attention(q, k2, v2, 0, 0.7, 4)[4:8], o[4:8]) and not torch.allclose(P.chunked_softmax_attention(q, k2, v2, 0, 0.7, 5)[4], o[4])
    # chunks are counted from position 0, not from where a portion starts
    assert torch.allclose(P.chunked_softmax_attention(q[6:], k, v, 6, 0.7, 4), o[6:])
    # rotation: entries 2i and 2i + 1 turn, products depend on the distance only, the factor of the scaling enters squared
    rot = {"base": 50.0, "dims": 6, "scaling": {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0}}
    a, b = torch.randn(1, 1, 10, dtype=P.F64), torch.randn(1, 1, 10, dtype=P.F64)
    ra, rb, rc, rd = (P.rotate_interleaved(x, p, rot) for x, p in ((a, 17), (b, 12), (a, 105), (b, 100)))
    assert torch.equal(ra[..., 6:], a[..., 6:]) and abs(float((ra * rb).sum() - (rc * rd).sum())) < 1e-9
    mult = 0.1 * math.log(4.0) + 1.0
    assert abs(float(ra[0, 0, 2:4].norm() / a[0, 0, 2:4].norm()) - mult) < 1e-12
    f, _ = P.rotary_table(rot)
    f0 = [50.0 ** (-2.0 * i / 6) for i in range(3)]
    assert f[0] == f0[0] and abs(f[1] / f0[1] - 0.625) < 1e-12 and abs(f[2] / f0[2] - 0.25) < 1e-12   # kept, half way up the ramp, slowed
    assert P.rotary_table({"base": 50.0, "dims": 6}) == (f0, 1.0)


def test_oracle_streams_delta_rule_and_norms():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=P.F64)
    mix = torch.tensor([[1.0, 2.0], [0.0, 3.0]], dtype=P.F64)   # [from, to]: stream 1 receives 2 x_0 + 3 x_1
    Y = P.write_streams(X, torch.tensor([[100.0, 0.0]], dtype=P.F64), mix, torch.tensor([1.0, -1.0], dtype=P.F64))
    assert Y[:, 0].tolist() == [[101.0, 2.0], [-68.0, 64.0]]
    assert P.read_streams(X, torch.tensor([3.0, -0.5], dtype=P.F64)).tolist() == [[-2.0, -4.0]]
    # one stream with coefficients 1 is the plain residual sum
    one = torch.ones(1, dtype=P.F64)
    assert torch.equal(P.write_streams(X[:1], X[1], one[:, None], one)[0], X[0] + X[1])
    g = torch.Generator().manual_seed(3)
    S, k, v = torch.randn(2, 4, 3, generator=g, dtype=P.F64), torch.randn(2, 4, generator=g, dtype=P.F64), torch.randn(2, 3, generator=g, dtype=P.F64)
    k = k / k.norm(dim=-1, keepdim=True)
    dec = torch.rand(2, 4, generator=g, dtype=P.F64)
    # beta 1 and a unit key: what is read at that key right after the write is the value itself, whatever the state held
    S1, o = P.delta_step(S, k, k, v, torch.ones(2, dtype=P.F64), dec)
    assert torch.allclose(o, v)
    # beta 0: only the decay acts, on the rows of key channels
    S0, o0 = P.delta_step(S, k, k, v, torch.zeros(2, dtype=P.F64), dec)
    assert torch.allclose(S0, dec[:, :, None] * S) and torch.allclose(o0[1], (dec[1] * k[1]) @ S[1])
    # convolution: the last tap multiplies the current row, the history carries over
    u, w, st = torch.arange(1.0, 7.0, dtype=P.F64)[:, None], torch.tensor([[100.0, 10.0, 1.0]], dtype=P.F64), {}
    assert torch.cat([P.short_conv(u[:2], w, st, "c"), P.short_conv(u[2:], w, st, "c")])[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]
    x = torch.randn(3, 8, generator=g, dtype=P.F64)
    assert torch.allclose((P.rms_norm(x, torch.ones(8, dtype=P.F64), 0.0) ** 2).mean(-1), torch.ones(3, dtype=P.F64))
