"""Vegilix through libssdk (HybridRunner / LLM) against the plain float64 oracle of tests/vegilix_plain.py, on small random
checkpoints of sizes of their own.  float32 storage is the sharp comparison (a wrong key, a window that is one position off, a
lost state or a kept key that is left out shows as an error of 1e-2 .. 1, rounding as 1e-6); bfloat16 runs are compared where
no discrete choice (expert routing) can flip."""
import copy

import numpy as np
import pytest
import torch

from tests import vegilix_util as U
from tests.vegilix_plain import PlainModel

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
    path = U.write_checkpoint(str(tmp_path / f"ckpt{seed}"), cfg, tensors)
    return _load(path, dtype, **kw), PlainModel(cfg, tensors), path


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _pages(n, block, first=0):
    return list(range(first, first + -(-n // block)))


def _per_pos(got, ref):
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def _portions(r, toks, sizes, slot, pages):
    out, pos, k = [], 0, 0
    while pos < len(toks):
        c = min(sizes[k % len(sizes)], len(toks) - pos)
        out.append(r.forward([(toks[pos:pos + c], pos, slot, pages, list(range(c)))])[0])
        pos, k = pos + c, k + 1
    return np.concatenate(out)


# both mixers, every feed-forward form and none, all sizes unequal: windows shorter and longer than a page and than the
# portions, no kept keys, a few, and more than a window; grouped heads 6:2, 4:4 and 5:1; full, partial and no rotation; value size above
# and below the key size; a loop over the middle of the program
FULL = [U.attention(mlp=U.moe()),
        U.retention(mlp=U.moe(experts=5, top=1, ff=12, shared_ff=0)),
        U.attention(heads=4, kv_heads=4, dim=8, vdim=5, window=40, keep=0, scale=0.5, dims=8, scaling=None, diff=0.2),
        U.retention(heads=2, dim=6, vdim=9, dims=0, decay=[0.5, 0.97], mlp=U.moe(experts=7, top=4, ff=12, shared_ff=20)),
        U.attention(heads=5, kv_heads=1, dim=6, vdim=3, window=9, keep=20, scale=0.6, dims=0, diff=0.7, mlp=U.moe(experts=3, top=3)),
        U.retention(heads=1, dim=5, vdim=33, dims=4, decay=[1.0])]
LOOP = (1, 4, 2)


@pytest.mark.parametrize("layer", [U.attention(), U.attention(heads=3, kv_heads=3, dim=12, vdim=12, window=0, dims=12),
                                   U.attention(heads=8, kv_heads=2, dim=4, vdim=7, window=1, keep=0, dims=2, diff=0.0),
                                   U.attention(heads=2, kv_heads=1, dim=33, vdim=40, window=16, keep=16, dims=0),
                                   U.attention(heads=1, kv_heads=1, dim=16, vdim=300, window=5, keep=1, dims=16),
                                   U.attention(heads=4, kv_heads=2, dim=9, vdim=6, window=8, keep=100, scaling=None)],
                         ids=["grouped", "no-groups-no-window", "window-of-one", "no-rotation-wide-values", "one-head-very-wide-values", "everything-kept"])
def test_attention_alone(tmp_path, layer):
    cfg = U.config([layer])
    r, plain, _ = _runner(tmp_path, cfg)
    toks = _tokens(53, cfg["vocab"], 1)
    lg, _, res = r.forward([(toks, 0, 2, _pages(53, 16, 5), list(range(53)))], residual=True)
    lo = []
    ref = plain.run(toks, layers_out=lo)
    assert U.rel_err(res[0], lo[0].numpy()) < F32_TOL
    assert U.rel_err(lg, ref.numpy()) < F32_TOL
    got = _portions(r, toks, [20, 2, 1, 1], 1, _pages(53, 16, 20))
    assert U.rel_err(got, ref.numpy()) < F32_TOL


@pytest.mark.parametrize("layer", [U.retention(), U.retention(heads=1, dim=1, vdim=1, dims=0, decay=[0.9]), U.retention(heads=2, dim=70, vdim=130, dims=70),
                                   U.retention(heads=5, dim=8, vdim=16, dims=8, decay=[0.0, 1e-3, 0.5, 0.999, 1.0]), U.retention(heads=2, dim=260, vdim=5, dims=2)],
                         ids=["ragged", "scalar-state", "several-tiles", "decays-from-zero-to-one", "tall-state"])
def test_retention_alone(tmp_path, layer):
    """More rows than a chunk, chunks that portions cut anywhere, then single tokens."""
    cfg = U.config([layer])
    r, plain, _ = _runner(tmp_path, cfg)
    n = 150
    toks = _tokens(n, cfg["vocab"], 1)
    lg, _, res = r.forward([(toks, 0, 2, _pages(n, 16, 5), list(range(n)))], residual=True)
    lo = []
    ref = plain.run(toks, layers_out=lo)
    assert U.rel_err(res[0], lo[0].numpy()) < F32_TOL
    assert U.rel_err(lg, ref.numpy()) < F32_TOL
    assert U.rel_err(_portions(r, toks, [65, 2, 64, 1, 1, 3], 1, _pages(n, 16, 20)), ref.numpy()) < F32_TOL


@pytest.mark.parametrize("mlp", [U.moe(), U.moe(experts=4, top=1, shared_ff=0), U.moe(experts=9, top=9, ff=12, shared_ff=20), U.moe(experts=2, top=2, ff=70, shared_ff=5),
                                 U.moe(experts=1, top=1, ff=3, shared_ff=1)], ids=["moe", "top1-no-shared", "all-chosen", "two-experts", "one-expert"])
def test_feed_forward_alone(tmp_path, mlp):
    """The mixer is switched off by a zero output projection; what is left of the layer is the normed feed-forward."""
    cfg = U.config([U.retention(mlp=mlp)])
    tensors = U.random_tensors(cfg, 3)
    tensors["l0.mix.o"].zero_()
    r, plain, _ = _runner(tmp_path, cfg, tensors=tensors, max_tokens=256, num_blocks=8, max_model_len=128)
    toks = _tokens(90, cfg["vocab"], 4)
    _, _, res = r.forward([(toks, 0, 0, _pages(90, 16), list(range(90)))], residual=True)
    lo = []
    plain.run(toks, layers_out=lo)
    assert U.rel_err(res[0], lo[0].numpy()) < F32_TOL


def test_every_tensor_carries_weight(tmp_path):
    """The comparison rests on every part of the layers: an oracle with one tensor changed is far from the engine."""
    cfg = U.config([U.attention(mlp=U.moe()), U.retention(mlp=U.moe())])
    r, plain, _ = _runner(tmp_path, cfg, seed=6)
    tensors = U.random_tensors(cfg, 6)
    toks = _tokens(60, cfg["vocab"], 2)
    lg, _ = r.forward([(toks, 0, 0, _pages(60, 16), list(range(60)))])
    assert U.rel_err(lg, plain.run(toks).numpy()) < F32_TOL
    names = [n for n in tensors if n not in ("embed", "head") and not any(f".e{k}." in n for k in range(1, 6))]
    assert len(names) > 30
    for name in names:
        other = {k: v.clone() for k, v in tensors.items()}
        other[name] = other[name].flip(0) if other[name].dim() == 1 else other[name] * 1.5 + 0.1
        assert U.rel_err(lg, PlainModel(cfg, other).run(toks).numpy()) > 10 * F32_TOL, name
    swapped = {k: v.clone() for k, v in tensors.items()}   # the two maps of every head exchanged
    for s in ("q", "k"):
        w = swapped[f"l0.mix.{s}"]
        swapped[f"l0.mix.{s}"] = w.view(-1, 2, 10, 40).flip(1).reshape(w.shape)
    assert U.rel_err(lg, PlainModel(cfg, swapped).run(toks).numpy()) > 10 * F32_TOL


def test_loop_equals_the_layers_written_out(tmp_path):
    """A looped program and one whose layers are copied out run the same kernels on the same numbers; every pass has rows and
    states of its own, also while decoding."""
    cfg = U.config(FULL[:4], loop=(1, 3, 3))
    tensors = U.random_tensors(cfg, 4)
    runs = [0, 1, 2, 1, 2, 1, 2, 3]
    flat = U.config([FULL[i] for i in runs])
    copies = {k: v for k, v in tensors.items() if not k.startswith("l")}
    for at, i in enumerate(runs):
        copies.update({f"l{at}." + k.split(".", 1)[1]: v for k, v in tensors.items() if k.startswith(f"l{i}.")})
    toks = _tokens(100, cfg["vocab"], 9)
    outs = []
    for c, t, seed in ((cfg, tensors, 4), (flat, copies, 5)):
        r, plain, _ = _runner(tmp_path, c, seed=seed, tensors=t)
        assert r.runs == (runs if c is cfg else list(range(8)))
        outs.append(_portions(r, toks, [60, 2, 1, 1, 1], 0, _pages(100, 16)))
        assert U.rel_err(outs[-1], plain.run(toks).numpy()) < F32_TOL
    assert np.array_equal(outs[0], outs[1])


def test_prefill_portions_and_token_by_token(tmp_path):
    cfg = U.config(FULL, loop=LOOP)
    r, plain, _ = _runner(tmp_path, cfg)
    n = 150
    toks = _tokens(n, cfg["vocab"], 5)
    ref = plain.run(toks).numpy()
    whole, _, res = r.forward([(toks, 0, 0, _pages(n, 16), list(range(n)))], residual=True)
    assert U.rel_err(whole, ref) < F32_TOL
    lo = []
    plain.run(toks, layers_out=lo)
    assert res.shape[0] == len(lo) == 9 and max(U.rel_err(a, b.numpy()) for a, b in zip(res, lo)) < F32_TOL
    # portions of several sizes, down to two tokens, cut inside pages, windows and chunks; then single tokens
    for sizes, slot, first in (([2, 3, 16, 5, 2, 31, 2, 17, 64], 1, 10), ([1], 2, 20), ([47, 2, 2, 2], 3, 30), ([65, 85], 0, 5)):
        got = _portions(r, toks, sizes, slot, _pages(n, 16, first))
        assert U.rel_err(got, ref) < F32_TOL
        assert np.abs(got - whole).max() < 1e-4 * np.abs(whole).max()


def test_batch_of_unequal_requests_equals_each_alone(tmp_path):
    cfg = U.config(FULL, loop=LOOP)
    r, plain, _ = _runner(tmp_path, cfg)
    lens = [110, 9, 33, 1]
    seqs = [_tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate(lens)]
    alone = [r.forward([(s, 0, 0, _pages(len(s), 16), list(range(len(s))))])[0] for s in seqs]
    # step 1: portions of requests 0, 1 and 2 + the whole of request 3; step 2: the rests, one of them a single token
    cut = [70, 8, 20, 1]
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
        # (a cut moves the chunks' borders and so the order of sums, nothing else)
        assert np.abs(g - alone[i]).max() < 2e-5 * np.abs(alone[i]).max(), f"request {i} depends on its batch"
        assert U.rel_err(g, plain.run(seqs[i]).numpy()) < F32_TOL


def test_pages_and_slots_are_reused(tmp_path, monkeypatch):
    """Requests come and go through the engine's managers: a later request gets the pages and the slot (the matrices of every
    pass) that an earlier one dirtied, in another order."""
    from ssd_b200.engine.block_manager import BlockManager
    from ssd_b200.engine.sequence import Sequence
    from ssd_b200.engine.state_manager import StateSlotManager
    cfg = U.config(FULL, loop=LOOP)
    r, plain, _ = _runner(tmp_path, cfg, num_blocks=8, n_slots=2)
    monkeypatch.setattr(Sequence, "block_size", 16)
    bm, sm = BlockManager(8, 16, prefix_reuse=False), StateSlotManager(2)
    prompts = [_tokens(n, cfg["vocab"], 20 + i) for i, n in enumerate([50, 40, 45, 30])]
    used_pages, used_slots, live = [], [], []
    for k, toks in enumerate(prompts):
        if len(live) == 2:  # the pools are full: the older request ends
            old = live.pop(0)
            bm.deallocate(old); sm.free(old)
        s = Sequence(toks)
        bm.allocate(s); sm.allocate(s)
        live.append(s)
        used_pages.append(tuple(s.block_table)); used_slots.append(s.state_slot)
        first = 1 if k == 3 else len(toks) // 2     # (a first portion of one token starts from a zero state too)
        a, _ = r.forward([(toks[:first], 0, s.state_slot, s.block_table, list(range(first)))])
        b, _ = r.forward([(toks[first:], first, s.state_slot, s.block_table, list(range(len(toks) - first)))])
        assert U.rel_err(np.concatenate([a, b]), plain.run(toks).numpy()) < F32_TOL, f"request {k}"
    assert len(set(used_slots)) < len(used_slots) and len({p for t in used_pages for p in t}) <= 8


@pytest.mark.parametrize("window,keep", [(23, 5), (32, 16), (150, 3), (30, 0)], ids=["inside-a-page-pair", "two-pages-one-kept", "hundreds-of-keys", "nothing-kept"])
def test_window_edges_with_sharp_attention(tmp_path, window, keep):
    """Attention made sharp: a large score scale puts nearly all weight on ONE visible key, wherever it lies — the oldest of the
    window, the last kept one — and never on a neighbour just outside.  In a prompt, in portions that start inside a window and while
    decoding over page borders.  The oracle with one more or one less key on either edge is far from the engine."""
    cfg = U.config([U.attention(heads=4, kv_heads=2, dim=8, vdim=8, window=window, keep=keep, scale=4.0, dims=4, mlp=U.moe())], mult=1.0)
    tensors = U.random_tensors(cfg, 7)
    r, plain, _ = _runner(tmp_path, cfg, seed=7, tensors=tensors, num_blocks=24, n_slots=2, max_model_len=384)
    n, tail = 330, 70
    toks = _tokens(n, cfg["vocab"], 8)
    ref = plain.run(toks).numpy()
    pages = list(range(23, 23 - 21, -1))
    out = [r.forward([(toks[:n - tail], 0, 0, pages, list(range(n - tail)))])[0]]
    for p in range(n - tail, n):  # decoding walks over four page borders
        out.append(r.forward([([toks[p]], p, 0, pages, [0])])[0])
    assert _per_pos(np.concatenate(out), ref).max() < 2e-3
    assert _per_pos(_portions(r, toks, [window + 3, 2, window - 1, 5, 64, 2], 1, pages), ref).max() < 2e-3
    for key, d in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1)):
        if key == "keep_first" and keep + d < 0:
            continue
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"][key] += d
        far = _per_pos(PlainModel(other, tensors).run(toks).numpy(), ref) > 0.02   # ten times the tolerance
        assert far[window:n - tail].sum() >= 3 and far[n - tail:].sum() >= 1, (key, d)


def _beacon_model(window, keep, dim, vdim):
    """One attention layer over one-hot tokens: token 1 is a beacon (its key of map 1 answers token 2's query of map 1 with a score
    far above all others), the rest is noise.  No rotation, so the score does not depend on the distance."""
    cfg = U.config([U.attention(heads=2, kv_heads=1, dim=dim, vdim=vdim, window=window, keep=keep, scale=1.5, dims=0, diff=0.3)], width=64, vocab=40, mult=2.0)
    t = U.one_hot_tensors(cfg, 12)
    u = torch.zeros(dim)
    u[3] = 1.0
    t["l0.mix.q.norm"].fill_(1.0); t["l0.mix.k.norm"].fill_(1.0)
    for tok in range(40):     # nobody else has anything along entry 3
        for name, heads in (("l0.mix.k", 2), ("l0.mix.q", 4)):
            v = torch.randn(heads, dim, generator=torch.Generator().manual_seed(100 + tok)) * 0.5
            v[:, 3] = 0.0
            U.set_token(t, name, tok, v.reshape(-1))
    beacon_k = torch.randn(2, dim, generator=torch.Generator().manual_seed(5)) * 0.2
    beacon_k[0] = 4.0 * u
    U.set_token(t, "l0.mix.k", 1, beacon_k.reshape(-1))
    query = torch.randn(4, dim, generator=torch.Generator().manual_seed(6)) * 0.2
    query[0] = query[2] = 4.0 * u
    U.set_token(t, "l0.mix.q", 2, query.reshape(-1))
    U.set_token(t, "l0.mix.v", 1, 8.0 * torch.randn(vdim, generator=torch.Generator().manual_seed(7)))
    return cfg, t


@pytest.mark.parametrize("dtype,dim,vdim", [("float32", 8, 16), ("bfloat16", 8, 16), ("bfloat16", 40, 96), ("bfloat16", 72, 128), ("bfloat16", 12, 20)])
def test_one_far_key_at_every_edge(tmp_path, dtype, dim, vdim):
    """A single key that outweighs hundreds of others, placed just inside and just outside the kept keys and the window, asked for
    by a prompt row, by a row of a two-token portion and by a decoded token."""
    window, keep = 90, 6
    cfg, tensors = _beacon_model(window, keep, dim, vdim)
    r, plain, _ = _runner(tmp_path, cfg, dtype=dtype, tensors=tensors, num_blocks=24, n_slots=2, max_model_len=384)
    tol = 2e-3 if dtype == "float32" else BF16_TOL
    noise = [3 + t % 37 for t in _tokens(300, 10 ** 6, 3)]
    pages = list(range(23, 1, -1))
    for beacon, asks in ((keep - 1, (200, 299)), (keep, (keep + window - 1, keep + window)), (0, (250,)), (127, (127 + window - 1, 127 + window)),
                         (128, (128 + window - 1, 128 + window, 290)), (200, (200 + window - 1, 200 + window))):
        toks = list(noise)
        toks[beacon] = 1
        for a in asks:
            toks[a] = 2
        state = plain.new_state()
        ref = plain.run(toks, state).numpy()
        hidden = list(noise)
        for a in asks:
            hidden[a] = 2
        without = plain.run(hidden).numpy()
        seen = [beacon < keep or a - beacon < window for a in asks]
        for a, s in zip(asks, seen):   # the beacon shows exactly where it is visible
            moved = U.rel_err(without[a], ref[a])
            assert (moved > 0.3) if s else (moved < 1e-9), (beacon, a)
        whole = r.forward([(toks, 0, 0, pages, list(range(300)))])[0]
        for a in asks:
            assert U.rel_err(whole[a], ref[a]) < tol, ("prompt", beacon, a)
            r.forward([(toks[:a - 1], 0, 1, pages, [])])
            two = r.forward([(toks[a - 1:a + 1], a - 1, 1, pages, [1])])[0]
            one = r.forward([([toks[a]], a, 1, pages, [0])])[0]     # (attention only: the row is simply written again)
            assert U.rel_err(two[0], ref[a]) < tol and U.rel_err(one[0], ref[a]) < tol, ("portion / decoded", beacon, a)


@pytest.mark.parametrize("dtype,dim,vdim", [("float32", 8, 6), ("bfloat16", 8, 6), ("bfloat16", 64, 128)])
def test_far_write_of_the_retention(tmp_path, dtype, dim, vdim):
    """One token writes, nothing decays, and the last of hundreds of positions reads it: over chunks, portions, pages and
    decoded tokens.  An oracle that lost the state at any border is far away."""
    cfg = U.config([U.retention(heads=2, dim=dim, vdim=vdim, dims=0, decay=[1.0, 0.999])], width=64, vocab=40, mult=2.0)
    t = U.one_hot_tensors(cfg, 13)
    u = torch.zeros(2, dim)
    u[:, 2] = 1.0
    for tok in range(40):
        for name in ("l0.mix.k", "l0.mix.q"):
            v = torch.randn(2, dim, generator=torch.Generator().manual_seed(200 + tok)) * 0.02
            v[:, 2] = 0.0
            U.set_token(t, name, tok, v.reshape(-1))
    U.set_token(t, "l0.mix.k", 1, 6.0 * u.reshape(-1))
    U.set_token(t, "l0.mix.q", 2, 6.0 * u.reshape(-1))
    r, plain, _ = _runner(tmp_path, cfg, dtype=dtype, tensors=t, num_blocks=30, n_slots=3, max_model_len=448)
    n, tol = 400, 1e-3 if dtype == "float32" else BF16_TOL
    toks = [3 + x % 37 for x in _tokens(n, 10 ** 6, 4)]
    toks[5] = 1
    toks[n - 1] = toks[270] = 2
    ref = plain.run(toks).numpy()
    forgot = list(toks)
    forgot[5] = 3
    assert U.rel_err(plain.run(forgot).numpy()[n - 1], ref[n - 1]) > 0.3
    pages = _pages(n, 16)
    whole = r.forward([(toks, 0, 0, pages, [270, n - 1])])[0]
    cut = _portions(r, toks, [64, 2, 65, 63, 7, 128], 1, pages)[[270, n - 1]]
    r.forward([(toks[:260], 0, 2, pages, [])])
    dec = _portions_from(r, toks, 260, 2, pages)[[10, n - 261]]
    for got in (whole, cut, dec):
        assert max(U.rel_err(got[i], ref[j]) for i, j in enumerate((270, n - 1))) < tol


def _portions_from(r, toks, pos0, slot, pages):
    return np.concatenate([r.forward([([toks[p]], p, slot, pages, [0])])[0] for p in range(pos0, len(toks))])


def test_decoding_sequences_of_unequal_context_share_a_step(tmp_path):
    """Three sequences decode together at contexts of a few, ~150 and ~300 tokens beside a prompt portion of a fourth, in one call:
    the single-token rows take the split-context attention and the one-pass retention, the portion its own kernels."""
    cfg = U.config([U.attention(heads=6, kv_heads=3, dim=8, vdim=10, window=200, keep=7, scale=2.0, mlp=U.moe()),
                    U.retention(heads=3, dim=8, vdim=12, decay=[0.9, 0.99, 0.999], mlp=U.moe()),
                    U.attention(heads=2, kv_heads=2, dim=6, vdim=6, window=8, keep=30, scale=2.0, dims=6)], loop=(0, 2, 2))
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
    cfg = U.config(FULL, loop=LOOP)
    r, plain, _ = _runner(tmp_path, cfg, seed=2)
    for n in (1, 2, 3, 4):   # below, at and beyond the kept keys
        toks = _tokens(n, cfg["vocab"], 30 + n)
        lg, _ = r.forward([(toks, 0, 1, [4], list(range(n)))])
        assert U.rel_err(lg, plain.run(toks).numpy()) < F32_TOL
    toks = _tokens(260, cfg["vocab"], 40)
    ref = plain.run(toks).numpy()
    out = [r.forward([(toks[:4], 0, 1, _pages(260, 16), [0, 1, 2, 3])])[0], _portions_from(r, toks, 4, 1, _pages(260, 16))]
    got = np.concatenate(out)
    assert _per_pos(got, ref).max() < 5 * F32_TOL, f"worst position {int(_per_pos(got, ref).argmax())}"


def test_long_batches_are_split_into_calls(tmp_path):
    cfg = U.config(FULL[:4], loop=(0, 2, 2))
    r, plain, _ = _runner(tmp_path, cfg, max_tokens=48, max_seqs=2, max_logit_rows=48)
    seqs = [_tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate([100, 7, 30])]
    lg, _ = r.forward([(s, 0, i, _pages(len(s), 16, 8 * i), [0, len(s) - 1]) for i, s in enumerate(seqs)])
    for i, s in enumerate(seqs):
        ref = plain.run(s).numpy()
        assert U.rel_err(lg[2 * i:2 * i + 2], ref[[0, len(s) - 1]]) < F32_TOL


def test_engine_rejects_what_it_cannot_serve(tmp_path):
    cfg = U.config([U.attention(heads=5, kv_heads=5)])
    tensors = U.random_tensors(cfg, 0)
    cfg["layers"][0]["mixer"]["kv_heads"] = 2      # 5 query heads do not split over 2 key/value heads
    with pytest.raises(RuntimeError):
        _load(U.write_checkpoint(str(tmp_path / "heads"), cfg, tensors))
    cfg = U.config([U.retention(heads=2, decay=[0.5, 1.5])])
    with pytest.raises(RuntimeError):              # a state that grows
        _load(U.write_checkpoint(str(tmp_path / "decay"), cfg, U.random_tensors(cfg, 0)))
    cfg = U.config([U.retention(heads=2, dim=8, dims=7)])
    with pytest.raises(RuntimeError):
        _load(U.write_checkpoint(str(tmp_path / "rot"), cfg, U.random_tensors(cfg, 0)))


@pytest.mark.parametrize("width", [40, 128, 36], ids=["rows-16B-aligned", "tcgen05-shapes", "unaligned"])
def test_bfloat16_storage(tmp_path, width):
    """bf16 weights / activations / cache with fp32 accumulation, residual, norms, router, scores and state.  Every expert
    is chosen (top == experts), so no routing decision can flip between the oracle and the rounded run.  The width picks
    the product kernel: 128 puts the dense projections on the tcgen05 GEMM, 40 on the mma.sync tile, 36 on the FMA tile."""
    every = dict(experts=4, top=4)
    cfg = U.config([U.attention(heads=4, kv_heads=2, dim=16, vdim=32, window=50, keep=5, dims=8, mlp=U.moe(**every)),
                    U.retention(heads=2, dim=16, vdim=24, dims=16, mlp=U.moe(**every)),
                    U.attention(heads=4, kv_heads=1, dim=24, vdim=16, window=20, keep=0, dims=24)], width=width, loop=(0, 2, 2))
    r, plain, _ = _runner(tmp_path, cfg, dtype="bfloat16")
    n = 120
    toks = _tokens(n, cfg["vocab"], 60)
    ref = plain.run(toks).numpy()
    whole, _ = r.forward([(toks, 0, 0, _pages(n, 16), list(range(n)))])
    assert U.rel_err(whole, ref) < BF16_TOL
    got = _portions(r, toks, [2, 30, 3, 64, 2] + [1] * 19, 1, _pages(n, 16, 9))
    assert U.rel_err(got, whole) < 2e-2


@pytest.mark.parametrize("dim,vdim,groups", [(8, 16, 1), (32, 32, 2), (40, 64, 4), (64, 104, 1), (24, 128, 3), (104, 72, 2), (128, 128, 16)])
def test_attention_on_the_tensor_cores(tmp_path, monkeypatch, dim, vdim, groups):
    """Every tile size of the fused two-map kernels, groups of 1 .. 16 heads, sharp scores, prompts of two sequences and decoding:
    against the path of separate products and a softmax (same rounded operands) and against the oracle."""
    cfg = U.config([U.attention(heads=2 * groups, kv_heads=2, dim=dim, vdim=vdim, window=70, keep=9, scale=2.0 / dim ** 0.5, dims=dim // 2 // 2 * 2)], width=64)
    tensors = U.random_tensors(cfg, 0)
    path = U.write_checkpoint(str(tmp_path / "tc"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    seqs = [_tokens(230, cfg["vocab"], 80), _tokens(131, cfg["vocab"], 81)]
    got = {}
    for on in ("1", "0"):
        monkeypatch.setenv("SSDK_HYB_GQA_MMA", on)
        r = _load(path, "bfloat16", num_blocks=64)
        pages = [_pages(230, 16, 30), _pages(131, 16, 3)]
        lg, _ = r.forward([(s[:-3], 0, i, p, list(range(len(s) - 3))) for i, (s, p) in enumerate(zip(seqs, pages))])
        dec = [r.forward([([s[len(s) - k]], len(s) - k, i, p, [0]) for i, (s, p) in enumerate(zip(seqs, pages))])[0] for k in (3, 2, 1)]
        got[on] = [np.concatenate([lg[:227]] + [d[0:1] for d in dec]), np.concatenate([lg[227:]] + [d[1:2] for d in dec])]
        r.close()
    for i, s in enumerate(seqs):
        assert U.rel_err(got["1"][i], plain.run(s).numpy()) < BF16_TOL
        assert U.rel_err(got["1"][i], got["0"][i]) < 2.5e-2


@pytest.mark.parametrize("dim,vdim", [(8, 8), (32, 64), (31, 100), (64, 32), (64, 64), (48, 128), (128, 16), (72, 64), (128, 128), (97, 33)])
def test_retention_on_the_tensor_cores(tmp_path, monkeypatch, dim, vdim):
    """Every tile size of the chunk kernels: the split products against plain fp32 FMA (same inputs: nearly equal) and the oracle."""
    cfg = U.config([U.retention(heads=3, dim=dim, vdim=vdim, dims=dim // 2 * 2, decay=[0.7, 0.98, 0.999])], width=64)
    tensors = U.random_tensors(cfg, 0)
    path = U.write_checkpoint(str(tmp_path / "tc"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    seqs = [_tokens(230, cfg["vocab"], 80), _tokens(131, cfg["vocab"], 81), _tokens(2, cfg["vocab"], 82)]
    got = {}
    for on in ("1", "0"):
        monkeypatch.setenv("SSDK_HYB_RETENTION_MMA", on)
        r = _load(path, "bfloat16", num_blocks=64)
        pages = [_pages(230, 16, 30), _pages(131, 16, 3), [0]]
        a, _, ra = r.forward([(s[:n], 0, i, p, []) for i, (s, p, n) in enumerate(zip(seqs, pages, (100, 1, 1)))], residual=True)
        b, _, rb = r.forward([(s[n:], n, i, p, []) for i, (s, p, n) in enumerate(zip(seqs, pages, (100, 1, 1)))], residual=True)
        got[on] = [np.concatenate([ra[0, :100], rb[0, :130]]), np.concatenate([ra[0, 100:101], rb[0, 130:260]]), np.concatenate([ra[0, 101:], rb[0, 260:]])]
        r.close()
    for i, s in enumerate(seqs):
        lo = []
        plain.run(s, layers_out=lo)
        assert U.rel_err(got["1"][i], lo[0].numpy()) < BF16_TOL
        assert U.rel_err(got["1"][i], got["0"][i]) < 2e-3


def test_bfloat16_calls_of_many_rows(tmp_path, monkeypatch):
    """More rows than one tile of the tcgen05 GEMM holds (256) and enough routed rows for the grouped tcgen05 expert GEMM; windows
    shorter than the prompts.  Two prompts of unequal length in one call, against the oracle, against portions, and against the
    mma.sync tile on the same checkpoint."""
    every = dict(experts=3, top=3, ff=64, shared_ff=64)
    cfg = U.config([U.attention(heads=4, kv_heads=2, dim=32, vdim=64, window=130, keep=4, dims=16, mlp=U.moe(**every)),
                    U.retention(heads=4, dim=32, vdim=32, dims=32, mlp=U.moe(**every))], width=128, vocab=96, loop=(0, 2, 2))
    tensors = U.random_tensors(cfg, 0)
    path = U.write_checkpoint(str(tmp_path / "rows"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    seqs = [_tokens(330, cfg["vocab"], 80), _tokens(271, cfg["vocab"], 81)]
    refs = [plain.run(s).numpy() for s in seqs]
    got = {}
    for tc in ("1", "0"):
        monkeypatch.setenv("SSDK_HYB_TC_EXPERTS", tc)
        r = _load(path, "bfloat16", max_tokens=1024, num_blocks=64)
        lg, _ = r.forward([(s, 0, i, _pages(len(s), 16, 30 * i), list(range(len(s)))) for i, s in enumerate(seqs)])
        got[tc] = [lg[:330], lg[330:]]
        for g, ref in zip(got[tc], refs):
            assert U.rel_err(g, ref) < BF16_TOL
        if tc == "1":
            assert U.rel_err(_portions(r, seqs[0], [200, 100, 30], 2, _pages(330, 16, 30)), got[tc][0]) < 2e-2
        r.close()
    assert U.rel_err(got["1"][0], got["0"][0]) < 1e-2


def test_greedy_generation_through_llm(tmp_path):
    """The public entry point: LLM.generate with the engine's scheduler (three prompts, two sequences at a time: the third
    waits and gets used pages and a used slot), temperature 0, against the oracle's greedy continuation."""
    from ssd_b200 import LLM, SamplingParams
    cfg = U.config(FULL[:4], vocab=64, loop=(1, 3, 2))
    tensors = U.random_tensors(cfg, 11)
    path = U.write_checkpoint(str(tmp_path / "gen"), cfg, tensors)
    plain = PlainModel(cfg, tensors)
    prompts = [_tokens(n, cfg["vocab"], 70 + i) for i, n in enumerate([21, 5, 40])]
    llm = LLM(path, dtype="float32", kvcache_block_size=16, max_model_len=128, max_num_batched_tokens=128, max_num_seqs=2)
    try:
        outs, _ = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True), use_tqdm=False)
    finally:
        llm.exit()
    for p, o in zip(prompts, outs):
        assert o["token_ids"] == plain.greedy(p, 12)
