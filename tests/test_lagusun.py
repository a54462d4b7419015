"""Lagusun through the engine against the plain implementation (``plain_lagusun``).

Every test runs three ways: over the kernels' plain PyTorch twins on the CPU (the package's
parts, cache manager, step function and scheduler are the ones under test there), and on the GPU
over the CUDA kernels in float32 and in bfloat16.
"""

from __future__ import annotations

import json

import numpy as np
import pytest
import torch

import lagusun_cases as lc
import plain_lagusun as plain
from lagusun_cases import BACKENDS

F64 = torch.float64


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(lc.CASES))
def test_whole_prompt_decoding_and_portions(tmp_path, backend, name):
    """A whole prompt in one step, the same tokens one by one from the first on, and portions of
    several sizes down to two tokens (cut inside pages, windows, chunks and the kernels' tiles) all
    give the plain logits."""
    cfg, tensors, folder, page = lc.case_folder(tmp_path, name, dtype=lc.stored_dtype(backend))
    n = 70 if name != "wide" else 200
    tokens = lc.clear_tokens(cfg, tensors, n, seed=3, dtype=backend[1])
    want = lc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = lc.make_replayer(folder, backend, 4 * 256, page)
    want.check(lc.feed(rp, "whole", tokens, [n]), "whole prompt")
    want.check(lc.feed(rp, "single", tokens, [] if n <= 70 else [n - 50]), "token by token")
    want.check(lc.feed(rp, "cut", tokens, [2, 3, 2, 7, 16, 2, 5, 9, 2, 11]), "portions")
    want.check(lc.feed(rp, "cut2", tokens, [page + 1, 2 * page - 1, 2, 2, 33]), "portions across pages")
    if n > 130:
        want.check(lc.feed(rp, "cut3", tokens, [69, 2, 18, 2, 64, 17, 2]), "portions at the edges of windows and chunks")
    assert rp.engine.cache.n_live() == 0


@pytest.mark.parametrize("backend", BACKENDS)
def test_batches_of_unequal_requests(tmp_path, backend):
    """Four live requests of different lengths, portions beside single tokens, in a pool so small
    that pages and slots are used again: every request's logits are those it gets alone."""
    cfg, tensors, folder, page = lc.case_folder(tmp_path, "mixed", dtype=lc.stored_dtype(backend))
    lengths = [61, 9, 34, 1, 47, 22, 80]
    reqs = {f"r{i}": lc.clear_tokens(cfg, tensors, n, seed=10 + i, dtype=backend[1]) for i, n in enumerate(lengths)}
    want = {rid: lc.plain_logits(cfg, tensors, toks, backend[1]) for rid, toks in reqs.items()}
    rp = lc.make_replayer(folder, backend, 4 * 64, page, max_num_seqs=4)
    rng = np.random.default_rng(0)
    waiting, live, at, got = list(reqs), [], {}, {rid: [] for rid in reqs}
    step = 0
    while waiting or live:
        while waiting and len(live) < 4:
            rid = waiting.pop(0)
            live.append(rid)
            at[rid] = 0
        entries, end = [], []
        for rid in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                                     # left out of this step
            left = len(reqs[rid]) - at[rid]
            n = 1 if (at[rid] > len(reqs[rid]) // 2) else int(min(left, rng.choice([2, 3, 5, 8, 13, 24])))
            entries.append({"id": rid, "tokens": reqs[rid][at[rid]:at[rid] + n], "want": list(range(n))})
            at[rid] += n
            if at[rid] == len(reqs[rid]):
                end.append(rid)
        if not entries:
            continue
        out = rp.run_step({"step": step, "entries": entries, "end": end})
        rp.engine.cache.check_invariants()
        row = 0
        for e in entries:
            got[e["id"]].append(out[row:row + len(e["tokens"])])
            row += len(e["tokens"])
        live = [rid for rid in live if rid not in end]
        step += 1
    for rid in reqs:
        want[rid].check(np.concatenate(got[rid]), rid)
    assert rp.engine.cache.n_live() == 0


@pytest.mark.parametrize("backend", BACKENDS)
def test_long_decoding_in_a_pool_shorter_than_the_request(tmp_path, backend):
    """260 tokens, most decoded one by one (recorded steps on the GPU), through a pool that holds 64: every page that
    windows and chunks have passed goes back and is used again.  Then another request in the same slot and pages."""
    cfg, tensors, folder, page = lc.case_folder(tmp_path, "awkward", dtype=lc.stored_dtype(backend))
    tokens = lc.clear_tokens(cfg, tensors, 260, seed=3, dtype=backend[1])
    rp = lc.make_replayer(folder, backend, 64, page, max_num_seqs=1)
    lc.plain_logits(cfg, tensors, tokens, backend[1]).check(lc.feed(rp, "long", tokens, [5, 17, 2, 2]), "long decoding")
    again = lc.clear_tokens(cfg, tensors, 20, seed=4, dtype=backend[1])
    lc.plain_logits(cfg, tensors, again, backend[1]).check(lc.feed(rp, "again", again, [1, 1, 3]), "the slot's next request")
    rp.engine.cache.check_invariants()


def test_pages_of_chunks_are_given_back():
    """The cache manager's chunk groups: all pages before the chunk that the next token falls into go back, whether a
    chunk's edge is a page's edge or not; a request cannot be shortened into a chunk whose pages are gone."""
    from torchllms_b200.cache.manager import CacheError, CacheManager
    from torchllms_b200.parts.base import CacheNeed
    m = CacheManager([(CacheNeed("chunk", 1, 4, 10), None, None), (CacheNeed("full", 1, 4), None, None)], page_size=4, pool_tokens=64,
                     max_num_seqs=2, max_len=64, dtype=torch.float32, device="cpu", max_step_tokens=16)
    h = m.claim()
    held = []
    for n in range(1, 41):
        m.extend_many([(h, 1)])
        m.pass_window(h)
        m.check_invariants()
        first = n // 10 * 10 // 4                       # the page of the first token of the next token's chunk
        pages = m.pages_of(h, 0)
        assert [b for b, p in enumerate(pages) if p >= 0] == list(range(first, len(pages))), n
        held.append(sum(p >= 0 for p in pages))
        assert all(p >= 0 for p in m.pages_of(h, 1))
    assert max(held) <= 4 and m.groups[0].allocator.n_free == m.groups[0].allocator.n_pages - held[-1]
    with pytest.raises(CacheError):
        m.truncate(h, 35)                               # 35 lies in the chunk 30 .. 39, whose pages are gone
    h2 = m.claim()
    m.extend_many([(h2, 18)])
    m.pass_window(h2)
    m.truncate(h2, 12)                                  # still in the chunk 10 .. 19
    m.check_invariants()
    with pytest.raises(CacheError):
        m.truncate(h2, 9)
    need = CacheNeed("chunk", 1, 4, 10)
    assert need.covering(CacheNeed("chunk", 1, 4, 10)) == need
    assert need.covering(CacheNeed("window", 1, 4, 3)) == CacheNeed("window", 1, 4, 10)
    assert need.covering(CacheNeed("full", 1, 4)).kind == "full"


def test_layers_of_experts_as_one_matrix(tmp_path):
    """The form a decode batch takes on the GPU (every expert's up matrix and the shared expert's as one matrix,
    zeros where a token did not choose an expert), forced for every step over the kernels' twins: the same logits."""
    from torch_ops import TorchOps
    from torchllms_b200.engine.replay import Replayer
    cfg, tensors, folder, page = lc.case_folder(tmp_path, "mixed")
    tokens = lc.clear_tokens(cfg, tensors, 40, seed=2, dtype="float32")
    ops = TorchOps()
    ops.dense_experts = True
    rp = Replayer(folder, "float32", 256, page_size=page, device="cpu", ops=ops, max_num_seqs=2)
    lc.plain_logits(cfg, tensors, tokens, "float32").check(lc.feed(rp, "a", tokens, [17, 2]), "all experts as one matrix")


# ---------------------------------------------------------------- one mechanism at a time

MIXERS = {
    "chunks": lc.chunked(heads=4, kv_heads=2, dim=12, rot_dims=8, size=13),
    "chunks-of-a-page": lc.chunked(heads=2, kv_heads=1, dim=20, rot_dims=20, size=8, base=30.0),
    "chunk-beyond-the-prompt": lc.chunked(heads=3, kv_heads=3, dim=16, rot_dims=0, size=500),
    "window": lc.windowed(heads=4, kv_heads=2, dim=8, vdim=24, rot_dims=8, size=11),
    "window-of-a-page": lc.windowed(heads=6, kv_heads=2, dim=16, vdim=8, rot_dims=4, size=8, softcap=0.7),
    "window-beyond-the-prompt": lc.windowed(heads=2, kv_heads=1, dim=10, vdim=10, rot_dims=2, size=500, scaling=None, softcap=50.0),
    "window-of-one": lc.windowed(heads=2, kv_heads=2, dim=4, vdim=4, rot_dims=4, size=1),
}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("kind", list(MIXERS))
def test_each_mixer_alone(tmp_path, backend, kind):
    """One layer without a feed-forward: the mixer is all there is between the embedding and the head."""
    cfg = lc.config([MIXERS[kind]], width=40, vocab=53, groups=2)
    dtype = lc.stored_dtype(backend)
    tensors = lc.stored(lc.tensors_for(cfg, seed=len(kind), sharp=3.0 if backend[1] == "float32" else 1.0), dtype)
    if "beyond" in kind and cfg["layers"][0]["type"] == "attention_2":
        tensors["l0.mix.pb"] = tensors["l0.mix.pb"] - 2.0       # ninety weights that are not divided by their sum
    tokens = lc.tokens_for(cfg, 90, seed=5)
    want = lc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = lc.make_replayer(lc.write_folder(tmp_path, kind, cfg, tensors, dtype), backend, 256, 8)
    want.check(lc.feed(rp, "p", tokens, [90]), "prompt")
    want.check(lc.feed(rp, "d", tokens, [3]), "decoded")
    want.check(lc.feed(rp, "c", tokens, [2, 2, 31, 2, 9, 17, 2]), "portions")


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("loop", [None, (0, 1, 2), (1, 3, 3), (0, 3, 2), (2, 3, 1)])
def test_loops(tmp_path, backend, loop):
    """No loop, a loop over the first layer, over the last two, over all layers, and one that runs
    once: every pass has a cache of its own and starts from the product of stream and embedding output with its
    own row added, also after a layer that leaves a scaled sum pending."""
    cfg = lc.config([lc.windowed(mlp=None), lc.chunked(mlp=None), lc.windowed(heads=2, kv_heads=2, dim=8, vdim=8, rot_dims=6, size=9, mlp=None)],
                    width=40, vocab=53, scale=2.0, groups=5, loop=loop)
    dtype = lc.stored_dtype(backend)
    tensors = lc.stored(lc.tensors_for(cfg, seed=7), dtype)
    tokens = lc.tokens_for(cfg, 40, seed=6)
    exact = plain.forward(cfg, tensors, tokens)
    if loop is not None:
        # each half of the product and the row matter
        d = cfg["width"]
        for change in ("row", "stream", "embedding"):
            bare = {k: v.clone() for k, v in tensors.items()}
            if change == "row":
                bare["loop.step"][:] = 0.0
            else:
                bare["loop.in"][:, slice(0, d) if change == "stream" else slice(d, 2 * d)] = 0.0
            assert (plain.forward(cfg, bare, tokens) - exact).abs().max() > 0.05, change
    want = lc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = lc.make_replayer(lc.write_folder(tmp_path, "loop", cfg, tensors, dtype), backend, 128, 8)
    want.check(lc.feed(rp, "p", tokens, [40]), "prompt")
    want.check(lc.feed(rp, "c", tokens, [2, 9, 2, 17]), "portions and decoded")


def _marked(cfg, tensors, tokens, key_at: int, query_at: int):
    """Weights changed so that in the first layer the query at ``query_at`` scores the key at ``key_at`` far above all
    others: the embedding rows of the two tokens are large along one coordinate each, which the layer's query and key
    projections pass on to an unrotated coordinate of every head."""
    t = {k: v.clone() for k, v in tensors.items()}
    layer = cfg["layers"][0]
    m = layer["mixer"]
    dk, rot = m["dim"], m["rot"]["dims"]
    # the two tokens are unique in the sequence; their rows point along coordinates 0 and 1, which no other token's row has
    t["embed"][:, :2] = 0.0
    for tok, axis in ((tokens[key_at], 0), (tokens[query_at], 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, axis] = 6.0
    t["l0.norm1"] = torch.ones(cfg["width"])
    for name, axis, heads in (("q", 1, m["heads"]), ("k", 0, m["kv_heads"])):
        w = t[f"l0.mix.{name}"]
        w[:, axis] = 0.0
        for h in range(heads):
            w[h * dk + rot] = 0.0
            w[h * dk + rot, axis] = 2.0
            if layer["type"] == "attention_2":
                t[f"l0.mix.{name}.b"][h * dk + rot] = 0.0
            else:
                t[f"l0.mix.{name}.norm"][h * dk + rot] = 1.0
    if layer["type"] == "attention_2":
        t["l0.mix.pb"][:] = -6.0                       # ordinary scores count for little
    return t


SIZE = 21          # of the windows and chunks below; pages hold 8


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("kind,key_at,query_at,inside", [
    ("window", 40, 40 + SIZE - 1, True), ("window", 40, 40 + SIZE, False),
    ("window", 47, 47 + SIZE - 1, True), ("window", 48, 48 + SIZE, False),
    ("chunk", 2 * SIZE, 3 * SIZE - 1, True), ("chunk", 3 * SIZE - 1, 3 * SIZE, False),
    ("chunk", 2 * SIZE, 3 * SIZE, False), ("chunk", 2 * SIZE + 5, 2 * SIZE + 19, True)])
def test_keys_at_the_edges_of_windows_and_chunks(tmp_path, backend, kind, key_at, query_at, inside):
    """A key that one query would score far above all others, just inside and just outside its window or chunk, in a
    prompt, in portions cut at the edge, and with the query decoded alone.  The test first proves on the plain
    implementation that a mask which is one token off would move the query's logits."""
    layer = lc.windowed(heads=2, kv_heads=1, dim=12, vdim=8, rot_dims=4, size=SIZE, softcap=25.0, scale=1.0) if kind == "window" \
        else lc.chunked(heads=2, kv_heads=1, dim=12, rot_dims=4, size=SIZE, scale=1.0)
    cfg = lc.config([layer], width=32, vocab=120, scale=1.0, groups=2)
    dtype = lc.stored_dtype(backend)
    n = 90
    tokens = [int(x) for x in np.random.default_rng(5).permutation(120)[:n]]
    base = lc.tensors_for(cfg, seed=11)
    tensors = lc.stored(_marked(cfg, base, tokens, key_at, query_at), dtype)
    off = json.loads(json.dumps(cfg))       # another mask: the key on the other side of its edge
    off["layers"][0]["mixer"]["mask"]["size"] = {("window", True): SIZE - 1, ("window", False): SIZE + 1,
                                                 ("chunk", True): query_at - key_at, ("chunk", False): 4 * SIZE}[kind, inside]
    exact, moved = (plain.forward(c, tensors, tokens)[query_at] for c in (cfg, off))
    assert (exact - moved).abs().max() > 0.3, "the marked key does not matter"
    want = lc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = lc.make_replayer(lc.write_folder(tmp_path, "edge", cfg, tensors, dtype), backend, 2 * 96, 8, max_num_seqs=2)
    want.check(lc.feed(rp, "p", tokens, [n]), "prompt")
    want.check(lc.feed(rp, "d", tokens, [query_at]), "the query decoded alone")
    want.check(lc.feed(rp, "c", tokens, [key_at, 2, max(query_at - key_at - 3, 1), 2, 2]), "portions at the edge")


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("kind", ["window", "chunk"])
def test_a_far_key_at_a_pages_border(tmp_path, backend, kind):
    """A key hundreds of places back, at a page's last and first place, that one query must find among all the
    others inside a long window or chunk, in a prompt, in portions and when the query is decoded alone.  The test first
    proves on the plain implementation that losing that key moves the query's logits."""
    page, n = 8, 300
    layer = lc.windowed(heads=2, kv_heads=1, dim=12, vdim=8, rot_dims=4, size=290, softcap=25.0, scale=1.0) if kind == "window" \
        else lc.chunked(heads=2, kv_heads=1, dim=12, rot_dims=4, size=400, scale=1.0)
    cfg = lc.config([layer], width=32, vocab=400, scale=1.0, groups=4)
    dtype = lc.stored_dtype(backend)
    base = lc.tensors_for(cfg, seed=11)
    tokens = [int(x) for x in np.random.default_rng(5).permutation(400)[:n]]
    query_at = n - 3
    for key_at in (page * 3 - 1, page * 4):
        tensors = lc.stored(_marked(cfg, base, tokens, key_at, query_at), dtype)
        exact = plain.forward(cfg, tensors, tokens)
        lost = plain.forward(cfg, tensors, tokens[:key_at] + [tokens[key_at + 1]] + tokens[key_at + 1:])
        assert (exact[query_at] - lost[query_at]).abs().max() > 0.3, "the marked key does not matter: the test would say nothing"
        want = lc.plain_logits(cfg, tensors, tokens, backend[1])
        rp = lc.make_replayer(lc.write_folder(tmp_path, f"far{key_at}", cfg, tensors, dtype), backend, 2 * 320, page, max_num_seqs=2)
        want.check(lc.feed(rp, "p", tokens, [n]), "prompt")
        want.check(lc.feed(rp, "c", tokens, [key_at, 2, 100, n - key_at - 102 - 8]), "portions, the query decoded alone")


def _without(name: str, cfg, tensors, tokens, monkeypatch):
    """Plain logits with one mechanism left out."""
    with monkeypatch.context() as mp:
        if name == "sink":
            mp.setattr(plain, "softmax_with_zero_sink", lambda s, seen: torch.softmax(s.masked_fill(~seen, float("-inf")), -1))
        elif name == "score bias":
            mp.setattr(plain, "sigmoid_weights", lambda s, seen, b: torch.sigmoid(s).masked_fill(~seen, 0.0))
        elif name == "sigmoid":
            mp.setattr(plain, "sigmoid_weights", lambda s, seen, b: torch.softmax((s + b).masked_fill(~seen, float("-inf")), -1))
        elif name == "norm groups":
            mp.setattr(plain, "grouped_norm", lambda x, w, groups, eps: plain.unit_rms(x, eps) * w)
        elif name == "head and row norms":
            mp.setattr(plain, "unit_rms", lambda x, eps: x)
        elif name == "bands":
            mp.setattr(plain, "frequencies", lambda dims, base, scaling: [base ** (-2.0 * i / dims) for i in range(dims // 2)])
        elif name == "exact gelu":
            mp.setattr(plain, "erf_gelu", lambda z: 0.5 * z * (1.0 + torch.tanh(0.7978845608028654 * (z + 0.044715 * z ** 3))))
        elif name == "layer scales":
            tensors = {k: torch.ones_like(v) if k.split(".")[-1] in ("ls1", "ls2") else v for k, v in tensors.items()}
        elif name == "correction":
            tensors = {k: torch.zeros_like(v) if k.endswith("correction") else v for k, v in tensors.items()}
        return plain.forward(cfg, tensors, tokens)


@pytest.mark.parametrize("backend", BACKENDS)
def test_every_mechanism_shows(tmp_path, backend, monkeypatch):
    """A model in which leaving out any one mechanism (the sink, a head's score bias, sigmoid in place of softmax, the
    norm's groups, the norms of q, k and v, the bands of the frequencies, the layer scales, the choice's correction, the
    exact gelu) moves the plain logits: the engine holds to the real ones, from a sequence's first token on."""
    cfg = lc.config([lc.chunked(heads=3, kv_heads=1, dim=8, rot_dims=6, size=11, scale=1.0, mlp=lc.moe(5, 2, 16, scale=2.0, shared=12)),
                     lc.windowed(heads=2, kv_heads=1, dim=8, vdim=12, rot_dims=8, base=200.0, size=14, softcap=2.0, scale=1.0, mlp=None)],
                    width=24, vocab=61, scale=4.0, groups=3)
    dtype = lc.stored_dtype(backend)
    tensors = lc.tensors_for(cfg, seed=3)
    tensors["embed"][:, :8] *= 3.0                       # the groups differ in size
    tensors["l0.mlp.correction"] = torch.tensor([0.3, -0.2, 0.2, -0.3, 0.0])
    tensors["l1.mix.pb"] = torch.tensor([1.0, -2.0])
    tensors = lc.stored(tensors, dtype)
    tokens = lc.clear_tokens(cfg, tensors, 50, seed=8, dtype=backend[1])
    exact = plain.forward(cfg, tensors, tokens)
    for name in ("sink", "score bias", "sigmoid", "norm groups", "head and row norms", "bands", "layer scales", "correction"):
        assert (_without(name, cfg, tensors, tokens, monkeypatch) - exact).abs().max() > 0.05, name
    assert (_without("exact gelu", cfg, tensors, tokens, monkeypatch) - exact).abs().max() > 3e-4
    want = lc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = lc.make_replayer(lc.write_folder(tmp_path, "all", cfg, tensors, dtype), backend, 128, 4)
    want.check(lc.feed(rp, "p", tokens, [50]), "prompt")
    want.check(lc.feed(rp, "d", tokens, []), "token by token from the first")
    want.check(lc.feed(rp, "c", tokens, [1, 2, 3, 9]), "portions")


# ---------------------------------------------------------------- kernels against the plain functions

def _ops(backend):
    if backend[0] == "cpu":
        from torch_ops import TorchOps
        return TorchOps(), torch.device("cpu")
    from torchllms_b200.kernels import get_ops
    return get_ops(), torch.device("cuda")


def _dt(backend):
    return torch.bfloat16 if backend[1] == "bfloat16" else torch.float32


@pytest.mark.parametrize("backend", BACKENDS)
def test_grouped_norm_with_a_scaled_sum(backend):
    """The norm kernel: groups of several widths (some no multiple of four, more groups than warps), a pending sum in
    one piece or as partial sums, with and without a scale, all rows or picked ones."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(1)
    dt = _dt(backend)
    for dim, groups in ((48, 3), (44, 2), (512, 1), (640, 40), (2048, 4), (30, 5)):
        for T in (3, 40):
            w, ls = torch.randn(dim, generator=g), torch.randn(dim, generator=g)
            for delta in (None, torch.randn(T, dim, generator=g).to(dt), torch.randn(3, T, dim, generator=g)):
                for scale in (None, ls) if delta is not None and groups > 1 else (ls,):
                    h = torch.randn(T, dim, generator=g)
                    x = h.to(F64)
                    if delta is not None:
                        d = delta.to(F64).sum(0) if delta.dim() == 3 else delta.to(F64)
                        x = x + (d if scale is None else d * scale.to(F64))
                    exact = plain.grouped_norm(x, w.to(F64), groups, 1e-5)
                    tol = 2e-5 if dt == torch.float32 else 2e-2
                    on = lambda t: None if t is None else t.to(dev)
                    stream = h.to(dev)
                    pick = torch.tensor([T - 1, 0], dtype=torch.int32)
                    some = ops.rmsnorm(stream, on(delta), w.to(dev), 1e-5, out_dtype=dt, rows=pick.to(dev), groups=groups, delta_scale=on(scale))
                    torch.testing.assert_close(some.cpu().double(), exact[pick.long()], atol=tol, rtol=tol)
                    assert torch.equal(stream.cpu(), h)                       # picked rows leave the stream alone
                    got = ops.rmsnorm(stream, on(delta), w.to(dev), 1e-5, out_dtype=dt, groups=groups, delta_scale=on(scale))
                    torch.testing.assert_close(got.cpu().double(), exact, atol=tol, rtol=tol)
                    torch.testing.assert_close(stream.cpu().double(), x, atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("backend", BACKENDS)
def test_stream_join(backend):
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(2)
    dt = _dt(backend)
    for dim in (48, 30):
        h, e, row, ls = torch.randn(5, dim, generator=g), torch.randn(5, dim, generator=g), torch.randn(dim, generator=g), torch.randn(dim, generator=g)
        for delta in (None, torch.randn(5, dim, generator=g).to(dt), torch.randn(2, 5, dim, generator=g)):
            for scale in (None, ls):
                for r in (None, row):
                    stream = h.to(dev)
                    both, new = ops.stream_join(stream, None if delta is None else delta.to(dev), None if scale is None else scale.to(dev),
                                                e.to(dev), None if r is None else r.to(dev), out_dtype=dt)
                    x = h.clone()
                    if delta is not None:
                        d = delta.float().sum(0) if delta.dim() == 3 else delta.float()
                        x = x + (d if scale is None else d * scale)
                    tol = 1e-5 if dt == torch.float32 else 2e-2
                    torch.testing.assert_close(both.cpu().float(), torch.cat([x, e], 1), atol=tol, rtol=tol)
                    assert torch.equal(stream.cpu(), h)
                    assert torch.equal(new.cpu(), torch.zeros(5, dim) if r is None else row.expand(5, dim))


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("interleaved", [False, True])
def test_norms_around_the_rotation(backend, interleaved):
    """The kernel behind the input projection: biases, norms over whole rows and per head, both pairings, rotations over
    a part of a head, all of it and none, values that are keys, gates that ride along, partial sums, few tokens (heads
    spread over CTAs) and many."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(3)
    dt = _dt(backend)
    page = 4
    shapes = [(4, 2, 16, 24, 8, False, False, True, True, True, 3), (4, 2, 16, 16, 8, True, True, False, False, False, 0),
              (6, 1, 128, 128, 64, True, True, False, False, False, 0), (8, 2, 64, 128, 64, False, False, True, True, True, 8),
              (3, 3, 10, 6, 6, False, True, True, False, True, 2), (5, 1, 7, 7, 0, True, False, True, True, True, 0)]
    for H, G, d, dv, rot, same, row_norm, head_norm, v_norm, bias, extra in shapes:
        for T in (3, 300):
            nq, nk, nv = H * d, G * d, 0 if same else G * dv
            width = nq + nk + nv + extra
            proj = torch.randn(T, width, generator=g).to(dt)
            planes = proj.float()[None] * torch.tensor([0.25, 0.75])[:, None, None]
            b = torch.randn(width, generator=g) if bias else None
            qw, kw = (torch.randn(nq, generator=g), torch.randn(nk, generator=g)) if row_norm else (None, None)
            pos = torch.randint(0, 50, (T,), generator=g, dtype=torch.int32)
            ang = torch.rand(50, max(rot // 2, 1), generator=g) * 6.0
            table = torch.stack([ang.cos(), ang.sin()], -1).contiguous()
            slots = torch.randperm(400, generator=g)[:T].to(torch.int32)
            # float64, straight from the description
            x = proj.to(F64) + (0.0 if b is None else b.to(F64))
            q, k, v = x[:, :nq], x[:, nq:nq + nk], x[:, nq + nk:nq + nk + nv]
            v = (k if same else v).reshape(T, G, dv)
            if row_norm:
                q, k = plain.unit_rms(q, 1e-5) * qw.to(F64), plain.unit_rms(k, 1e-5) * kw.to(F64)
            def turn(y):
                y = y.clone()
                if rot:
                    u_at = slice(0, rot, 2) if interleaved else slice(0, rot // 2)
                    v_at = slice(1, rot, 2) if interleaved else slice(rot // 2, rot)
                    c, s = ang.to(F64).cos()[pos.long()][:, None], ang.to(F64).sin()[pos.long()][:, None]
                    a, e = y[..., u_at].clone(), y[..., v_at].clone()
                    y[..., u_at], y[..., v_at] = a * c - e * s, e * c + a * s
                return plain.unit_rms(y, 1e-5) if head_norm else y
            q, k = turn(q.reshape(T, H, d)), turn(k.reshape(T, G, d))
            if v_norm:
                v = plain.unit_rms(v, 1e-5)
            for src in (proj, planes):
                kp, vp = torch.zeros(100, G, page, d, dtype=dt, device=dev), torch.zeros(100, G, page, dv, dtype=dt, device=dev)
                on = lambda t: None if t is None else t.to(dev)
                got, gate = ops.norm_rope_store(
                    on(src), on(pos), on(table), n_q_heads=H, n_k_heads=G, head_dim=d, v_head_dim=dv, rot_dims=rot, interleaved=interleaved,
                    n_extra=extra, k_pages=kp, v_pages=vp, slot_mapping=on(slots), page_size=page, out_dtype=dt, bias=on(b),
                    values_are_keys=same, q_norm=on(qw), k_norm=on(kw), qk_head_norm=head_norm, v_head_norm=v_norm, eps=1e-5)
                tol = 3e-5 if dt == torch.float32 else 3e-2
                sl = slots.long()
                torch.testing.assert_close(got.cpu().double(), q, atol=tol, rtol=tol)
                torch.testing.assert_close(kp.cpu().double()[sl // page, :, sl % page], k, atol=tol, rtol=tol)
                torch.testing.assert_close(vp.cpu().double()[sl // page, :, sl % page], v, atol=tol, rtol=tol)
                if extra:
                    torch.testing.assert_close(gate.cpu().double(), torch.sigmoid(x[:, nq + nk + nv:]), atol=tol, rtol=tol)
                untouched = torch.ones(400, dtype=torch.bool)
                untouched[sl] = False
                rest = untouched.nonzero().flatten()
                assert not kp.cpu()[rest // page, :, rest % page].any() and not vp.cpu()[rest // page, :, rest % page].any()


@pytest.mark.parametrize("backend", BACKENDS)
def test_attention_weights_and_masks(backend):
    """The attention kernels with chunks and windows, a zero sink and sigmoid weights with a bias per head and a cap:
    prompt portions that cross edges, decode steps with keys split over CTAs, sizes for the tensor-core kernel and
    sizes it does not take, against the score matrices written out."""
    ops, dev = _ops(backend)
    dt = _dt(backend)
    g = torch.Generator().manual_seed(4)
    page = 8
    for H, G, d, dv in ((4, 2, 16, 24), (6, 3, 96, 96), (2, 1, 36, 20), (8, 1, 136, 128)):
        for lens, past in (([5, 33, 1], [0, 7, 300]), ([1, 1], [700, 41]), ([70], [90])):
            T, kv = sum(lens), [p + n for p, n in zip(past, lens)]
            n_pages = sum(-(-k // page) for k in kv) + 1
            keys = [torch.randn(k, G, d, generator=g).to(dt) for k in kv]
            vals = [torch.randn(k, G, dv, generator=g).to(dt) for k in kv]
            q = torch.randn(T, H, d, generator=g).to(dt)
            bias = torch.randn(H, generator=g)
            for mask, weights, cap in (("chunk", "softmax", 0.0), ("window", "sigmoid", 2.0), ("chunk", "sigmoid", 0.0), ("window", "softmax", 1.5)):
                for size in (1, 13, 64, 350):
                    k_pages = torch.full((n_pages, G, page, d), float("nan")).to(dt)         # what is not visible must not be read into a result
                    v_pages = torch.full((n_pages, G, page, dv), float("nan")).to(dt)
                    table = torch.full((len(lens), max(-(-k // page) for k in kv)), -1, dtype=torch.int32)
                    at = 1
                    want = torch.zeros(T, H, dv, dtype=F64)
                    row = 0
                    for b, (n, p0, k) in enumerate(zip(lens, past, kv)):
                        first = max(0, p0 - size + 1) if mask == "window" else p0 // size * size
                        for j in range(first // page, -(-k // page)):
                            table[b, j] = at
                            k_pages[at], v_pages[at] = 0.0, 0.0
                            m = min(page, k - j * page)
                            k_pages[at, :, :m], v_pages[at, :, :m] = keys[b][j * page:j * page + m].transpose(0, 1), vals[b][j * page:j * page + m].transpose(0, 1)
                            at += 1
                        seen = (plain.near_past(k, size) if mask == "window" else plain.same_chunk(k, size))[p0:]
                        for h in range(H):
                            s = q[row:row + n, h].to(F64) @ keys[b][:, h // (H // G)].to(F64).T * d ** -0.5
                            if cap:
                                s = cap * torch.tanh(s / cap)
                            w = plain.sigmoid_weights(s, seen, bias[h].to(F64)) if weights == "sigmoid" else plain.softmax_with_zero_sink(s, seen)
                            want[row:row + n, h] = w @ vals[b][:, h // (H // G)].to(F64)
                        row += n
                    q_start = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
                    kw = {"window": size if mask == "window" else None, "chunk": size if mask == "chunk" else None, "weights": weights}
                    if weights == "sigmoid":
                        kw["score_bias"] = bias.to(dev)
                    else:
                        kw["sinks"] = torch.zeros(H, device=dev)
                    got = ops.paged_attention(q.to(dev), k_pages.to(dev), v_pages.to(dev), table.to(dev), q_start.to(dev),
                                              torch.tensor(kv, dtype=torch.int32).to(dev), n_seqs=len(lens), max_q_len=max(lens),
                                              max_kv_len=max(kv), scale=d ** -0.5, page_size=page, softcap=cap, **kw)
                    tol = 5e-5 if dt == torch.float32 else 2e-2
                    torch.testing.assert_close(got.cpu().double(), want, atol=tol * max(1.0, float(want.abs().max())), rtol=tol,
                                               msg=lambda m: f"{(H, G, d, dv)} {lens} {past} {mask} {size} {weights}: {m}")


@pytest.mark.parametrize("backend", BACKENDS)
def test_router_with_a_correction(backend):
    """The correction steers the choice and leaves the weights alone; weights are normalised and scaled."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(0)
    for E, top in ((10, 2), (7, 1), (8, 8), (64, 6)):
        for T in (5, 70):
            x = torch.randn(T, 16, generator=g).to(_dt(backend))
            w, corr = torch.randn(E, 16, generator=g), 0.5 * torch.randn(E, generator=g)
            chosen, weights = plain.route(x.to(F64) @ w.to(F64).T, corr.to(F64), {"experts": E, "top": top, "scale": 1.7})
            got_c, got_w, _ = ops.moe_route(x.to(dev), w.to(dev), corr.to(dev), n_experts=E, top=top, scale=1.7, renormalize=True,
                                            shared_gate=False, score="sigmoid", renorm_eps=1e-20)
            order, got_order = chosen.sort(-1), got_c.cpu().long().sort(-1)
            assert torch.equal(order.values, got_order.values), (E, top, T)
            torch.testing.assert_close(got_w.cpu().double().gather(1, got_order.indices), weights.gather(1, order.indices), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("backend", BACKENDS)
def test_exact_gelu(backend):
    ops, dev = _ops(backend)
    x = torch.linspace(-6.0, 6.0, 1000)[None].repeat(2, 1).to(_dt(backend))
    got = ops.activation(x.to(dev), "gelu").cpu().double()
    want = plain.erf_gelu(x.to(F64))
    if _dt(backend) == torch.float32:
        torch.testing.assert_close(got, want, atol=1e-6, rtol=1e-6)
    else:        # one rounding to bfloat16, also far out on the negative side (apart from an absolute 1e-6)
        torch.testing.assert_close(got, want, atol=1e-6, rtol=2.0 ** -8)


def test_frequencies_by_band():
    """The engine's table against the plain frequencies, with wavelengths in all three bands and on both borders."""
    import math
    from torchllms_b200.parts.rope import precise_rotary_table
    for dims, base, band in ((16, 500.0, lc.BAND), (8, 3.0, {"factor": 2.0, "low": 1.0, "high": 1.0, "original": 10}),
                             (64, 10000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}), (6, 20.0, None)):
        f = plain.frequencies(dims, base, band)
        if band and dims == 16:
            lengths = [2 * math.pi * base ** (2.0 * i / dims) for i in range(dims // 2)]
            assert any(l < 40 / 3 for l in lengths) and any(40 / 3 < l < 40 for l in lengths) and any(l > 40 for l in lengths)
        table = precise_rotary_table(dims, base, 1.0, 100, band=band)
        ang = torch.arange(100, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)
        torch.testing.assert_close(table.double(), torch.stack([ang.cos(), ang.sin()], -1), atol=1e-6, rtol=1e-6)


# ---------------------------------------------------------------- configuration, loading, generation

def test_configuration_and_names(tmp_path):
    """The configuration's errors name their key; a folder with a tensor too many or too few is refused;
    the configuration is written back as it was read."""
    from torch_ops import TorchOps
    from torchllms_b200.config.model_config import ConfigError
    from torchllms_b200.config.registry import load_config
    from torchllms_b200.engine.loading import load_model
    from torchllms_b200.models import lagusun
    from torchllms_b200.weights.loader import WeightError
    cfg, tensors, folder, _page = lc.case_folder(tmp_path, "mixed")
    _arch, parsed = load_config(folder)
    assert parsed.to_hf() == json.loads((folder / "config.json").read_text())
    assert [r[0] for r in parsed.runs()] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and [r[1] for r in parsed.runs()][1::3] == [0, 1, 2, None]
    for path, value, word in ((("layers", 0, "mixer", "softcap"), 0, "softcap"), (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 2, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 1, "mixer", "vdim"), 6, "vdim"),
                              (("layers", 1, "mixer", "mask", "size"), 0, "mask.size"), (("norm", "groups"), 5, "norm.groups"),
                              (("layers", 0, "mixer", "rot", "scaling", "low"), 9.0, "rot.scaling"),
                              (("layers", 0, "mlp", "router", "top"), 7, "top"), (("layers", 0, "mlp", "kind"), "dense", "kind"),
                              (("loop", "stop"), 9, "loop"), (("loop", "times"), 0, "loop"),
                              (("layers", 0, "type"), "conv", "type"), (("embedding",), None, "embedding")):
        bad = json.loads(json.dumps(cfg))
        node = bad
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            lagusun.parse_config(bad, "test")
    for change in ("extra", "missing"):
        t = dict(tensors)
        if change == "extra":
            t["l1.mix.v"] = torch.zeros(32, 48)
        else:
            del t["l0.mix.pb"]
        with pytest.raises(WeightError):
            load_model(lc.write_folder(tmp_path, change, cfg, t), dtype="float32", device="cpu", ops=TorchOps())


@pytest.mark.parametrize("backend", BACKENDS)
def test_greedy_generation_through_the_scheduler(tmp_path, backend):
    """``LLM.generate`` (scheduler, sampler, look-ahead) against a plain greedy loop."""
    from torchllms_b200.inference import LLM
    cfg, tensors, folder, page = lc.case_folder(tmp_path, "mixed")
    kw = {}
    if backend[0] == "cpu":
        from torch_ops import TorchOps
        kw = dict(ops=TorchOps())
    llm = LLM(folder, max_len=128, max_bsz=3, device=backend[0], precision=backend[1], page_size=page,
              max_num_batched_tokens=24, **kw)
    prompts = [lc.clear_tokens(cfg, tensors, n, seed=20 + n, dtype=backend[1]) for n in (3, 30, 11, 1)]
    results = llm.generate(prompt_token_ids=prompts, temperature=0.0, max_new_tokens=12, disable_tqdm=True)
    compared = 0
    for prompt, r in zip(prompts, results):
        seq = list(prompt)
        for _ in range(12):
            margins: list = []
            logits = plain.forward(cfg, tensors, seq, margins_out=margins)[-1]
            top = torch.topk(logits, 2).values
            if min((float(m.min()) for m in margins), default=1.0) < (1e-4 if backend[1] == "float32" else 0.01):
                break                         # a close call in routing may fall either way: stop comparing this request
            token, tie = r.token_ids[len(seq) - len(prompt)], 1e-3 if backend[1] == "float32" else 0.15
            if float(top[0] - top[1]) < tie:  # and so may a near tie of the logits
                assert float(top[0] - logits[token]) < tie
            else:
                assert token == int(torch.argmax(logits))
                compared += 1
            seq.append(token)
        assert r.error is None and len(r.token_ids) == 12
    assert compared >= (30 if backend[1] == "float32" else 4)


def test_random_weights_mode_writes_a_folder_that_loads(tmp_path):
    """The framework's random-weights mode for this architecture: a folder under the checkpoint's
    names that loads like any other, and the same model built without a file."""
    from torchllms_b200.config.registry import load_config
    from torchllms_b200.engine.loading import load_model, random_model
    from torchllms_b200.weights.random_init import write_random_model
    from torchllms_b200.weights.safetensors_io import TensorSource
    from torch_ops import TorchOps
    _cfg, _tensors, folder, _page = lc.case_folder(tmp_path, "mixed")
    _arch, parsed = load_config(folder)
    out = write_random_model(tmp_path / "random", parsed, seed=3)
    names = set(TensorSource(out).names())
    assert {"embed", "head", "final.norm", "loop.in", "loop.step", "l0.mix.pb", "l0.mix.v.b", "l1.mix.q.norm", "l0.mlp.e5.up",
            "l0.mlp.shared.down", "l0.mlp.correction", "l4.ls2"} <= names
    assert not {"l1.mix.v", "l1.norm2", "l1.ls2", "l4.mlp.shared.up", "l2.mix.q.norm"} & names
    _, _, from_file = load_model(out, dtype="float32", device="cpu", ops=TorchOps())
    _, _, direct = random_model(parsed, 3, dtype="float32", device="cpu", ops=TorchOps())
    assert torch.equal(from_file.embedding, direct.embedding) and torch.equal(from_file.head, direct.head)
