"""Vatolorn through libssdk (HybridRunner / LLM) against the plain float64 oracle of tests/vatolorn_plain.py, on small random
checkpoints of sizes of their own.  float32 storage is the sharp comparison (a wrong key, a chunk edge that is one position
off, a lost state or a transposed stream mixture shows as an error of 1e-2 .. 1, rounding as 1e-6)."""
import copy

import numpy as np
import pytest
import torch

from tests import vatolorn_util as U
from tests.vatolorn_plain import PlainModel

pytestmark = pytest.mark.gpu

F32_TOL = 3e-4
BF16_TOL = 6e-2


def _load(path, dtype="float32", **kw):
    from ssd_b200.hybrid import HybridRunner, HybridSpec, load_hybrid_weights
    spec = HybridSpec.from_dir(path)
    w = load_hybrid_weights(path, spec, {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype], "cuda:0")
    args = dict(dtype=dtype, max_tokens=512, max_seqs=4, block_size=16, num_blocks=40, n_slots=4, max_model_len=512)
    args.update(kw)
    return HybridRunner(spec, w, **args)


def _runner(tmp_path, cfg, seed=0, dtype="float32", tensors=None, **kw):
    tensors = tensors if tensors is not None else U.random_tensors(cfg, seed)
    path = U.write(str(tmp_path / f"ckpt{seed}"), cfg, tensors)
    return _load(path, dtype, **kw), PlainModel(cfg, tensors), path


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _pages(n, block, first=0):
    return list(range(first, first + -(-n // block)))


def _per_pos(got, ref):
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


# all sizes unequal, chunks shorter and longer than a page and than the portions, 1 .. 5 taps, grouped heads 3:1, 1:1 and 5:1 on
# both sides, full, partial, unscaled and no rotation, values wider and narrower than keys, ranks above and below 8
FULL = [U.parallel(mlp=U.dense()),
        U.parallel(U.attention(heads=4, kv_heads=4, dim=8, vdim=12, conv=1, chunk=40, scale=0.5, dims=8, scaling=None),
                   U.delta(heads=2, kv_heads=2, dim=5, vdim=9, conv=1, decay_rank=8, gate_rank=1), mlp=U.dense(ff=64)),
        U.parallel(U.attention(heads=5, kv_heads=1, dim=6, vdim=3, conv=5, chunk=7, scale=0.6, dims=0),
                   U.delta(heads=4, kv_heads=1, dim=20, vdim=3, conv=5, decay_rank=17, gate_rank=4)),
        U.parallel(U.attention(heads=2, kv_heads=1, dim=16, vdim=16, conv=2, chunk=64, dims=4),
                   U.delta(heads=3, kv_heads=3, dim=40, vdim=36, conv=2, decay_rank=3, gate_rank=16), mlp=U.dense(ff=33))]


@pytest.mark.parametrize("left", [U.attention(), U.attention(heads=4, dim=12, vdim=8, conv=4, dims=8), U.attention(heads=4, dim=8, vdim=20, conv=2, dims=8), U.attention(heads=3, kv_heads=3, dim=12, vdim=12, conv=1, chunk=1000, dims=12),
                                  U.attention(heads=8, kv_heads=2, dim=4, vdim=7, conv=6, chunk=1, dims=2, scaling=None),
                                  U.attention(heads=2, kv_heads=1, dim=33, vdim=40, conv=2, chunk=16, dims=0),
                                  U.attention(heads=1, kv_heads=1, dim=7, vdim=1, conv=3, chunk=5, dims=6, base=10.0),
                                  U.attention(conv=0, chunk=0)],
                         ids=["grouped", "whole-vectors-4-taps", "whole-vectors-2-taps", "no-groups-full-rotation-wide-chunk", "chunk-of-one", "no-rotation-wide-values", "one-head-odd-size", "no-conv-no-chunks"])
def test_attention_alone(tmp_path, left):
    """The delta rule's norm weight is zero, so the layer is the attention half behind the streams."""
    cfg = U.config([U.parallel(left=left, right=U.delta(heads=4, kv_heads=2, vdim=8))], streams=2)
    tensors = U.random_tensors(cfg, 1)
    tensors["l0.mix.right.out"].zero_()
    r, plain, _ = _runner(tmp_path, cfg, tensors=tensors)
    toks = _tokens(37, cfg["vocab"], 1)
    lg, _, res = r.forward([(toks, 0, 2, _pages(37, 16, 5), list(range(37)))], residual=True)
    lo = []
    ref = plain.run(toks, layers_out=lo)
    assert U.rel_err(res[0], lo[0].numpy()) < F32_TOL and U.rel_err(lg, ref.numpy()) < F32_TOL


# key sizes on every form of the scan: one to eight 16-byte pieces per lane, 4 / 8 / 16 lanes per column, whole vectors and
# ragged ones, and the form that keeps the column in shared memory; many columns (four lanes each) and few (eight)
@pytest.mark.parametrize("right", [U.delta(), U.delta(heads=1, kv_heads=1, dim=16, vdim=64, conv=1, decay_rank=1, gate_rank=1),
                                   U.delta(heads=5, kv_heads=1, dim=3, vdim=33, conv=6), U.delta(heads=4, kv_heads=2, dim=32, vdim=20, conv=2),
                                   U.delta(heads=2, kv_heads=2, dim=64, vdim=8), U.delta(heads=2, kv_heads=1, dim=50, vdim=6),
                                   U.delta(heads=2, kv_heads=2, dim=100, vdim=12), U.delta(heads=1, kv_heads=1, dim=77, vdim=5),
                                   U.delta(heads=2, kv_heads=1, dim=200, vdim=4), U.delta(heads=1, kv_heads=1, dim=300, vdim=8),
                                   U.delta(heads=2, kv_heads=1, dim=520, vdim=40), U.delta(heads=80, kv_heads=20, dim=40, vdim=64),
                                   U.delta(heads=80, kv_heads=80, dim=72, vdim=64)],
                         ids=["grouped", "wide-values", "tiny-keys", "32", "64", "50", "100", "77", "200", "300", "520", "many-columns-40", "many-columns-72"])
def test_delta_rule_alone(tmp_path, right):
    """The attention's norm weight is zero, so the layer is the delta-rule half; a prompt in portions, then single tokens."""
    cfg = U.config([U.parallel(right=right)], streams=2)
    tensors = U.random_tensors(cfg, 2)
    tensors["l0.mix.left.out"].zero_()
    r, plain, _ = _runner(tmp_path, cfg, tensors=tensors)
    toks = _tokens(45, cfg["vocab"], 2)
    ref, out, pos = plain.run(toks).numpy(), [], 0
    for c in [33, 2, 5] + [1] * 5:
        out.append(r.forward([(toks[pos:pos + c], pos, 2, _pages(45, 16, 5), list(range(c)))])[0])
        pos += c
    assert _per_pos(np.concatenate(out), ref).max() < F32_TOL


@pytest.mark.parametrize("streams,width,ff", [(1, 40, 28), (2, 36, 64), (4, 33, 7), (5, 48, 96), (8, 64, 20), (11, 40, 28), (3, 35, 50)])
def test_streams_and_feed_forward(tmp_path, streams, width, ff):
    """Every form of the streams' step (registers for 1, 2, 4, 8 or up to 32 streams, vectors or single channels), with and
    without a feed-forward in the layer."""
    cfg = U.config([U.parallel(mlp=U.dense(ff)), U.parallel(), U.parallel(mlp=U.dense(ff + 4))], streams=streams, width=width)
    r, plain, _ = _runner(tmp_path, cfg, seed=streams, max_tokens=128, num_blocks=8, max_model_len=128)
    toks = _tokens(50, cfg["vocab"], 4)
    lg, _, res = r.forward([(toks, 0, 0, _pages(50, 16), list(range(50)))], residual=True)
    lo = []
    ref = plain.run(toks, layers_out=lo)
    for i in range(3):
        assert U.rel_err(res[i], lo[i].numpy()) < F32_TOL
    assert U.rel_err(lg, ref.numpy()) < F32_TOL


def test_every_part_carries_weight(tmp_path):
    """The comparison rests on every part of the layer: an oracle with one of them changed is far from the engine."""
    left = U.attention(dim=18, dims=16, base=30.0, scaling={"factor": 3.0, "original": 300, "fast": 8.0, "slow": 1.0})
    cfg = U.config([U.parallel(left=copy.deepcopy(left), mlp=U.dense()), U.parallel(left=copy.deepcopy(left), mlp=U.dense())], streams=3)
    tensors = U.random_tensors(cfg, 6)
    r, plain, _ = _runner(tmp_path, cfg, tensors=tensors)
    toks = _tokens(60, cfg["vocab"], 2)
    lg, _ = r.forward([(toks, 0, 0, _pages(60, 16), list(range(60)))])
    assert U.rel_err(lg, plain.run(toks).numpy()) < F32_TOL

    def swap(name):
        def f(t):
            t[name] = t[name].T.contiguous()
        return f

    def last_tap(name):
        def f(t):
            t[name].zero_()
            t[name][:, -1] = 1.0
        return f

    changes = {"mixture of the streams, to and from swapped": swap("l0.hc1.mix"), "feed-forward's mixture swapped": swap("l1.hc2.mix"),
               "stream reading": lambda t: t["l1.hc1.in"].fill_(1 / 3), "stream writing": lambda t: t["l0.hc2.out"].fill_(0.8),
               "query bias": lambda t: t["l0.mix.left.q.b"].zero_(), "value bias": lambda t: t["l0.mix.left.v.b"].zero_(),
               "key convolution": last_tap("l0.mix.left.k.conv"), "delta key convolution": last_tap("l0.mix.right.k.conv"),
               "query norm weight": lambda t: t["l0.mix.left.q.norm"].fill_(1.0), "key norm weight": lambda t: t["l0.mix.left.k.norm"].fill_(1.0),
               "decay per channel": lambda t: t["l0.mix.right.a2"].zero_(), "decay bias": lambda t: t["l0.mix.right.dt_bias"].fill_(-0.7),
               "decay rate": lambda t: t["l0.mix.right.A_log"].fill_(-1.0), "output gate": lambda t: t["l0.mix.right.g2"].zero_(),
               "beta": lambda t: t["l0.mix.right.b"].zero_(), "head norm": lambda t: t["l0.mix.right.norm"].fill_(1.0),
               "left result's norm": lambda t: t["l0.mix.left.out"].fill_(1.0), "right result's norm": lambda t: t["l0.mix.right.out"].fill_(1.0)}
    for name, change in changes.items():
        other = {k: v.clone() for k, v in tensors.items()}
        change(other)
        assert U.rel_err(lg, PlainModel(cfg, other).run(toks).numpy()) > 10 * F32_TOL, name
    for key, val in (("logit_scale", 0.75), ("norm", {"eps": 3e-2})):
        assert U.rel_err(lg, PlainModel(dict(cfg, **{key: val}), tensors).run(toks).numpy()) > 10 * F32_TOL, key
    for path, val in ((("rot", "base"), 200.0), (("rot", "scaling", "factor"), 2.0), (("rot", "scaling", "original"), 150), (("rot", "scaling", "fast"), 3.0),
                      (("rot", "scaling", "slow"), 4.0), (("scale",), 0.5), (("mask", "size"), 25)):
        other = copy.deepcopy(cfg)
        for lc in other["layers"]:
            d = lc["mixer"]["left"]
            for k in path[:-1]:
                d = d[k]
            d[path[-1]] = val
        assert U.rel_err(lg, PlainModel(other, tensors).run(toks).numpy()) > 3 * F32_TOL, path


def test_prefill_portions_and_token_by_token(tmp_path):
    cfg = U.config(FULL, streams=3)
    r, plain, _ = _runner(tmp_path, cfg)
    n = 150
    toks = _tokens(n, cfg["vocab"], 5)
    ref = plain.run(toks).numpy()
    whole, _ = r.forward([(toks, 0, 0, _pages(n, 16), list(range(n)))])
    assert U.rel_err(whole, ref) < F32_TOL
    # portions of several sizes, down to two tokens (shorter than the taps), cut inside pages and chunks; then single tokens
    for sizes, slot, first in (([2, 3, 16, 5, 2, 31, 2, 17, 64], 1, 10), ([1] * n, 2, 20), ([47, 2, 2, 2], 3, 30)):
        out, pos, k = [], 0, 0
        while pos < n:
            c = min(sizes[k % len(sizes)], n - pos)
            out.append(r.forward([(toks[pos:pos + c], pos, slot, _pages(n, 16, first), list(range(c)))])[0])
            pos, k = pos + c, k + 1
        got = np.concatenate(out)
        assert U.rel_err(got, ref) < F32_TOL
        assert np.abs(got - whole).max() < 1e-4 * np.abs(whole).max()


def test_batch_of_unequal_requests_equals_each_alone(tmp_path):
    cfg = U.config(FULL)
    r, plain, _ = _runner(tmp_path, cfg)
    lens = [70, 9, 33, 1]
    seqs = [_tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate(lens)]
    alone = [r.forward([(s, 0, 0, _pages(len(s), 16), list(range(len(s))))])[0] for s in seqs]
    # step 1: portions of requests 0, 1 and 2 + the whole of request 3; step 2: the rests, one of them a single token
    cut = [40, 8, 20, 1]
    pages = [_pages(n, 16, 8 * i) for i, n in enumerate(lens)]
    a, _ = r.forward([(seqs[i][:cut[i]], 0, i, pages[i], list(range(cut[i]))) for i in range(4)])
    b, _ = r.forward([(seqs[i][cut[i]:], cut[i], i, pages[i], list(range(lens[i] - cut[i]))) for i in (2, 1, 0)])
    got = {i: [] for i in range(4)}
    o = 0
    for i in range(4):
        got[i].append(a[o:o + cut[i]]); o += cut[i]
    o = 0
    for i in (2, 1, 0):
        got[i].append(b[o:o + lens[i] - cut[i]]); o += lens[i] - cut[i]
    for i in range(4):
        g = np.concatenate(got[i])
        assert np.abs(g - alone[i]).max() < 1e-5 * np.abs(alone[i]).max(), f"request {i} depends on its batch"
        assert U.rel_err(g, plain.run(seqs[i]).numpy()) < F32_TOL


def test_pages_and_slots_are_reused(tmp_path, monkeypatch):
    """Requests come and go through the engine's managers: a later request gets the pages and the slot (delta matrices,
    convolution histories of every layer) that an earlier one dirtied, in another order."""
    from ssd_b200.engine.block_manager import BlockManager
    from ssd_b200.engine.sequence import Sequence
    from ssd_b200.engine.state_manager import StateSlotManager
    cfg = U.config(FULL, streams=2)
    r, plain, _ = _runner(tmp_path, cfg, num_blocks=8, n_slots=2)
    monkeypatch.setattr(Sequence, "block_size", 16)
    bm, sm = BlockManager(8, 16, prefix_reuse=False), StateSlotManager(2)
    used_pages, used_slots, live = [], [], []
    for k, n in enumerate([50, 40, 45, 30]):
        toks = _tokens(n, cfg["vocab"], 20 + k)
        if len(live) == 2:  # the pools are full: the older request ends
            old = live.pop(0)
            bm.deallocate(old); sm.free(old)
        s = Sequence(toks)
        bm.allocate(s); sm.allocate(s)
        live.append(s)
        used_pages.append(tuple(s.block_table)); used_slots.append(s.state_slot)
        half = n // 2
        a, _ = r.forward([(toks[:half], 0, s.state_slot, s.block_table, list(range(half)))])
        b, _ = r.forward([(toks[half:], half, s.state_slot, s.block_table, list(range(n - half)))])
        assert U.rel_err(np.concatenate([a, b]), plain.run(toks).numpy()) < F32_TOL, f"request {k}"
    assert len(set(used_slots)) < len(used_slots) and len({p for t in used_pages for p in t}) <= 8


@pytest.mark.parametrize("chunk", [23, 32, 150], ids=["inside-a-page-pair", "two-pages", "hundreds-of-keys"])
def test_chunk_edges_with_sharp_attention(tmp_path, chunk):
    """Attention made sharp: a large score scale puts nearly all weight on ONE key of the chunk, wherever it lies — also on
    the chunk's first key, and never on the one just before it.  In a prompt, in portions that start inside a chunk and while
    decoding over page and chunk borders.  The oracle with chunks of one position more or less is far from the engine, so
    the comparison does rest on the edge."""
    cfg = U.config([U.parallel(U.attention(heads=4, kv_heads=2, dim=8, vdim=8, conv=2, chunk=chunk, scale=4.0, dims=4), mlp=U.dense()),
                    U.parallel(U.attention(heads=3, kv_heads=3, dim=8, vdim=8, conv=1, chunk=chunk + 9, scale=4.0, dims=8))])
    tensors = U.random_tensors(cfg, 7)
    r, plain, _ = _runner(tmp_path, cfg, seed=7, tensors=tensors, num_blocks=24, n_slots=2, max_model_len=384)
    n, tail = 330, 70
    toks = _tokens(n, cfg["vocab"], 8)
    ref = plain.run(toks).numpy()
    pages = list(range(23, 23 - 21, -1))
    out = [r.forward([(toks[:n - tail], 0, 0, pages, list(range(n - tail)))])[0]]
    for p in range(n - tail, n):  # decoding walks over four page borders and at least one chunk border
        out.append(r.forward([([toks[p]], p, 0, pages, [0])])[0])
    assert _per_pos(np.concatenate(out), ref).max() < 2e-3, f"worst position {int(_per_pos(np.concatenate(out), ref).argmax())}"
    # portions that start in the middle of a chunk, end at its edge, and span several chunks
    out, pos = [], 0
    for c in [chunk + 3, 2, chunk - 5, 5, 64, 2, 400]:
        c = min(c, n - pos)
        if c:
            out.append(r.forward([(toks[pos:pos + c], pos, 1, pages, list(range(c)))])[0])
        pos += c
    assert pos == n and _per_pos(np.concatenate(out), ref).max() < 2e-3
    for li in (0, 1):
        for d in (-1, 1):
            other = copy.deepcopy(cfg)
            other["layers"][li]["mixer"]["left"]["mask"]["size"] += d
            far = _per_pos(PlainModel(other, tensors).run(toks).numpy(), ref) > 0.02   # ten times the tolerance
            assert far.sum() >= 3, (li, d)


def test_far_write_of_the_delta_rule_is_kept(tmp_path):
    """One token writes into key channels that never decay and is read hundreds of positions later, over many chunks, pages and
    calls: beta, decay and key of that token are planted so that the value stands out."""
    d = U.delta(heads=2, kv_heads=1, dim=8, vdim=6, conv=1, decay_rank=4, gate_rank=4)
    cfg = U.config([U.parallel(U.attention(chunk=16), d)], streams=1, vocab=50)
    tensors = U.random_tensors(cfg, 12)
    p = "l0.mix.right."
    tensors[p + "A_log"].fill_(-9.0)      # g within 1e-4 of 1: nothing fades over the test
    tensors["l0.mix.left.out"].zero_()
    # all tokens but the two special ones write almost nothing (beta near 0): the embedding's first entry carries the write gate
    tensors["embed"][:, 0] = -3.0
    tensors["embed"][49, 0] = 3.0
    tensors[p + "b"].zero_()
    tensors[p + "b"][:, 0] = 20.0
    tensors["l0.norm1"].fill_(1.0)
    tensors["l0.hc1.in"].fill_(1.0)
    tensors = {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}
    r, plain, _ = _runner(tmp_path, cfg, seed=12, tensors=tensors)
    n = 400
    toks = [49 if i == 3 else t for i, t in enumerate(_tokens(n, 49, 13))]
    ref = plain.run(toks).numpy()
    other = plain.run([t if i != 3 else 7 for i, t in enumerate(toks)]).numpy()
    assert _per_pos(other, ref)[n - 50:].min() > 30 * F32_TOL        # the write is what the last positions read
    out, pos = [], 0
    for c in [2, 100, 3, 150, 45] + [1] * 100:
        out.append(r.forward([(toks[pos:pos + c], pos, 1, _pages(n, 16, 3), list(range(c)))])[0])
        pos += c
    assert pos == n and _per_pos(np.concatenate(out), ref).max() < F32_TOL


def test_decoding_sequences_of_unequal_context_share_a_step(tmp_path):
    """Three sequences decode together at contexts of a few, ~150 and ~300 tokens beside a prompt portion of a fourth: the
    single-token rows take the split-context attention over their chunks, the portion the GEMM path, in one call."""
    cfg = U.config([U.parallel(U.attention(heads=6, kv_heads=3, dim=8, vdim=10, chunk=200, scale=2.0), mlp=U.dense()),
                    U.parallel(U.attention(heads=2, kv_heads=2, dim=6, vdim=6, conv=4, chunk=8, scale=2.0), U.delta(heads=4, kv_heads=4, dim=24, vdim=16)),
                    U.parallel(U.attention(heads=2, kv_heads=1, dim=8, vdim=4, conv=3, chunk=1000, scale=1.0))], streams=4)
    r, plain, _ = _runner(tmp_path, cfg, seed=5, num_blocks=64)
    lens, steps = [3, 150, 300, 90], 6
    seqs = [_tokens(n + steps, cfg["vocab"], 90 + i) for i, n in enumerate(lens)]
    refs = [plain.run(s).numpy() for s in seqs]
    pages = [_pages(len(s), 16, first) for s, first in zip(seqs, (58, 40, 5, 30))]
    for i in range(3):  # prompts of the decoding sequences, each alone
        r.forward([(seqs[i][:lens[i]], 0, i, pages[i], [lens[i] - 1])])
    got = [[] for _ in seqs]
    for t in range(steps):
        ents = [([seqs[i][lens[i] + t]], lens[i] + t, i, pages[i], [0]) for i in range(3)]
        lo, hi = 16 * t, (16 * (t + 1) if t < steps - 1 else len(seqs[3]))
        ents.insert(1, (seqs[3][lo:hi], lo, 3, pages[3], list(range(hi - lo))))
        lg, _ = r.forward(ents)
        got[0].append(lg[0:1]); got[3].append(lg[1:1 + hi - lo]); got[1].append(lg[1 + hi - lo:2 + hi - lo]); got[2].append(lg[2 + hi - lo:])
    for i in range(3):
        assert U.rel_err(np.concatenate(got[i]), refs[i][lens[i]:]) < 2e-3, f"decoding sequence {i}"
    assert U.rel_err(np.concatenate(got[3]), refs[3]) < 2e-3


def test_first_tokens_and_long_decoding(tmp_path):
    cfg = U.config(FULL, streams=2)
    r, plain, _ = _runner(tmp_path, cfg, seed=2)
    for n in (1, 2, 3):   # fewer tokens than taps: the rest of the convolutions' reach is zeros, whatever the slot holds
        toks = _tokens(n, cfg["vocab"], 30 + n)
        lg, _ = r.forward([(toks, 0, 1, [4], list(range(n)))])
        assert U.rel_err(lg, plain.run(toks).numpy()) < F32_TOL
    toks = _tokens(260, cfg["vocab"], 40)
    ref = plain.run(toks).numpy()
    out = [r.forward([(toks[:4], 0, 1, _pages(260, 16), [0, 1, 2, 3])])[0]]
    for p in range(4, 260):
        out.append(r.forward([([toks[p]], p, 1, _pages(260, 16), [0])])[0])
    got = np.concatenate(out)
    assert _per_pos(got, ref).max() < 5 * F32_TOL, f"worst position {int(_per_pos(got, ref).argmax())}"


def test_long_batches_are_split_into_calls(tmp_path):
    cfg = U.config(FULL[:3])
    r, plain, _ = _runner(tmp_path, cfg, max_tokens=48, max_seqs=2, max_logit_rows=48)
    seqs = [_tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate([100, 7, 30])]
    lg, _ = r.forward([(s, 0, i, _pages(len(s), 16, 8 * i), [0, len(s) - 1]) for i, s in enumerate(seqs)])
    for i, s in enumerate(seqs):
        assert U.rel_err(lg[2 * i:2 * i + 2], plain.run(s).numpy()[[0, len(s) - 1]]) < F32_TOL


def test_engine_rejects_what_it_cannot_serve(tmp_path):
    cfg = U.config([U.parallel(U.attention(heads=5, kv_heads=5))])
    tensors = U.random_tensors(cfg, 0)
    cfg["layers"][0]["mixer"]["left"]["kv_heads"] = 2      # 5 query heads do not split over 2 key/value heads
    with pytest.raises(RuntimeError):
        _load(U.write(str(tmp_path / "heads"), cfg, tensors))
    cfg = U.config([U.parallel()], streams=33)
    tensors = U.random_tensors(cfg, 0)
    with pytest.raises(RuntimeError):
        _load(U.write(str(tmp_path / "streams"), cfg, tensors))


@pytest.mark.parametrize("width", [40, 128, 36], ids=["rows-16B-aligned", "tcgen05-shapes", "unaligned"])
def test_bfloat16_storage(tmp_path, width):
    """bf16 weights / activations / cache with fp32 accumulation, residual streams, norms, scores, decays and gates.  The
    width picks the product kernel: 128 puts the dense projections on the tcgen05 GEMM, 40 on the mma.sync tile, 36 on the
    FMA tile."""
    cfg = U.config([U.parallel(U.attention(heads=4, kv_heads=2, dim=16, vdim=16, chunk=50, dims=8),
                               U.delta(heads=4, kv_heads=2, dim=32, vdim=32, decay_rank=12, gate_rank=64), mlp=U.dense(ff=64)),
                    U.parallel(U.attention(heads=4, kv_heads=1, dim=16, vdim=24, conv=4, chunk=20, dims=16),
                               U.delta(heads=2, kv_heads=2, dim=20, vdim=64, decay_rank=64, gate_rank=10), mlp=U.dense(ff=192))], width=width, streams=3)
    r, plain, _ = _runner(tmp_path, cfg, dtype="bfloat16")
    n = 120
    toks = _tokens(n, cfg["vocab"], 60)
    ref = plain.run(toks).numpy()
    whole, _ = r.forward([(toks, 0, 0, _pages(n, 16), list(range(n)))])
    assert U.rel_err(whole, ref) < BF16_TOL
    out, pos = [], 0
    for c in [2, 30, 3, 64, 2] + [1] * 19:
        out.append(r.forward([(toks[pos:pos + c], pos, 1, _pages(n, 16, 9), list(range(c)))])[0])
        pos += c
    # single-token rows take the fused decode attention, which keeps its weights in fp32: equal up to bf16 rounding
    assert U.rel_err(np.concatenate(out), whole) < 2e-2


def test_bfloat16_calls_of_many_rows(tmp_path):
    """More rows than one tile of the tcgen05 GEMM holds (256), chunks of at least a block of query rows (128) and smaller
    ones, so that the portion path runs in several query blocks over shifted key ranges.  Two prompts of unequal length in one
    call, against the oracle and against portions."""
    cfg = U.config([U.parallel(U.attention(heads=4, kv_heads=2, dim=16, vdim=16, chunk=130, dims=16),
                               U.delta(heads=4, kv_heads=2, dim=64, vdim=64, decay_rank=64, gate_rank=64), mlp=U.dense(ff=192)),
                    U.parallel(U.attention(heads=2, kv_heads=2, dim=32, vdim=32, chunk=60, dims=16), mlp=U.dense(ff=64)),
                    U.parallel(U.attention(heads=2, kv_heads=1, dim=32, vdim=32, chunk=1000, dims=16))], width=128, vocab=96)
    tensors = U.random_tensors(cfg, 0)
    path = U.write(str(tmp_path / "rows"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    seqs = [_tokens(330, cfg["vocab"], 80), _tokens(271, cfg["vocab"], 81)]
    r = _load(path, "bfloat16", max_tokens=1024, num_blocks=64)
    lg, _ = r.forward([(s, 0, i, _pages(len(s), 16, 30 * i), list(range(len(s)))) for i, s in enumerate(seqs)])
    for g, s in zip((lg[:330], lg[330:]), seqs):
        assert U.rel_err(g, plain.run(s).numpy()) < BF16_TOL
    out, pos = [], 0
    for c in [200, 100, 30]:
        out.append(r.forward([(seqs[0][pos:pos + c], pos, 2, _pages(330, 16, 30), list(range(c)))])[0])
        pos += c
    assert U.rel_err(np.concatenate(out), lg[:330]) < 2e-2


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,chunk", [(6, 2, 40, 64, 50), (8, 2, 128, 96, 130), (3, 3, 72, 128, 1000), (16, 1, 24, 8, 77), (5, 1, 64, 16, 0)])
def test_attention_on_the_tensor_cores(tmp_path, monkeypatch, heads, kv_heads, dim, vdim, chunk):
    """bf16: the fused portion and decode kernels (every tile size, groups of one to sixteen heads, heads that do not fill a
    tile, chunks shorter and longer than a tile of keys) against the oracle and against the GEMM path.  Attention is sharp
    enough that a key too many or too few at a chunk's edge shows far above bf16 rounding."""
    att = U.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=2, chunk=chunk, scale=2.5 / dim ** 0.5, dims=8)
    cfg = U.config([U.parallel(copy.deepcopy(att)), U.parallel(copy.deepcopy(att), mlp=U.dense(ff=64))], width=64, vocab=96)
    tensors = U.random_tensors(cfg, 3)
    path = U.write(str(tmp_path / "mma"), cfg, tensors)
    n = 330
    toks = _tokens(n, cfg["vocab"], 15)
    ref, got = PlainModel(cfg, tensors).run(toks).numpy(), {}
    for mma in ("1", "0"):
        monkeypatch.setenv("SSDK_HYB_GQA_MMA", mma)
        r = _load(path, "bfloat16", num_blocks=64)
        pages = _pages(n, 16, 7)[::-1]
        whole, _ = r.forward([(toks, 0, 0, pages, list(range(n)))])
        out, pos = [], 0
        for c in [67, 2, 150, 1, 1, 60, 9] + [1] * 40:   # beside a second sequence's portion and a third one's single token
            ents = [(toks[pos:pos + c], pos, 1, pages, list(range(c))), (toks[:5], 0, 2, [40], [])]
            out.append(r.forward(ents + [([toks[0]], 0, 3, [41], [])])[0])
            pos += c
        got[mma] = (whole, np.concatenate(out))
        for g in got[mma]:
            assert U.rel_err(g, ref) < BF16_TOL and _per_pos(g, ref).max() < 5 * BF16_TOL
        r.close()
    assert U.rel_err(got["1"][0], got["0"][0]) < 2e-2 and U.rel_err(got["1"][1], got["0"][1]) < 2e-2
    if chunk:
        other = copy.deepcopy(cfg)
        for lc in other["layers"]:
            lc["mixer"]["left"]["mask"]["size"] += 1
        moved = _per_pos(PlainModel(other, tensors).run(toks).numpy(), ref)
        assert chunk > n or moved.max() > 5 * BF16_TOL


def test_gated_feed_forward_in_the_gemm(tmp_path, monkeypatch):
    """bf16: the gated feed-forward whose activation runs in the epilogue of the tcgen05 GEMM (a width of whole 64-column tiles,
    and one that ends inside a tile) against the separate activation kernel and the oracle: several row chunks, a short
    portion, single tokens."""
    cfg = U.config([U.parallel(mlp=U.dense(ff=1600)), U.parallel(mlp=U.dense(ff=1548))], width=128, streams=2)
    tensors = U.random_tensors(cfg, 0)
    path = U.write(str(tmp_path / "glu"), cfg, tensors)
    toks = _tokens(310, cfg["vocab"], 5)
    ref, got = PlainModel(cfg, tensors).run(toks).numpy(), {}
    for glu in ("1", "0"):
        monkeypatch.setenv("SSDK_HYB_TC_GLU", glu)
        r = _load(path, "bfloat16")
        out, pos = [], 0
        for c in [290, 17, 1, 1, 1]:
            out.append(r.forward([(toks[pos:pos + c], pos, 2, _pages(310, 16), list(range(c)))])[0])
            pos += c
        got[glu] = np.concatenate(out)
        assert U.rel_err(got[glu], ref) < BF16_TOL
        r.close()
    assert U.rel_err(got["1"], got["0"]) < 5e-3


def test_greedy_generation_through_llm(tmp_path):
    """The public entry point: LLM.generate with the engine's scheduler (three prompts, two sequences at a time: the third
    waits and gets used pages and a used slot), temperature 0, against the oracle's greedy continuation."""
    from ssd_b200 import LLM, SamplingParams
    cfg = U.config(FULL, vocab=64, streams=3)
    tensors = U.random_tensors(cfg, 11)
    path = U.write(str(tmp_path / "gen"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    prompts = [_tokens(n, cfg["vocab"], 70 + i) for i, n in enumerate([21, 5, 40])]
    llm = LLM(path, dtype="float32", kvcache_block_size=16, max_model_len=128, max_num_batched_tokens=128, max_num_seqs=2)
    try:
        outs, _ = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True), use_tqdm=False)
    finally:
        llm.exit()
    for p, o in zip(prompts, outs):
        assert o["token_ids"] == plain.greedy(p, 12)
