"""Bomotar through the engine against the plain implementation (``plain_bomotar``).

Every test runs three ways: over the kernels' plain PyTorch twins on the CPU (the package's
parts, cache manager, step function and scheduler are the ones under test there), and on the GPU
over the CUDA kernels in float32 and in bfloat16.
"""

from __future__ import annotations

import copy
import json

import numpy as np
import pytest
import torch

import bomotar_cases as bc
import plain_bomotar as plain
from bomotar_cases import BACKENDS

F64 = torch.float64


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(bc.CASES))
def test_whole_prompt_decoding_and_portions(tmp_path, backend, name):
    """A whole prompt in one step, the same tokens one by one from the first on, and portions of
    several sizes down to two tokens (cut inside pages, convolutions and the kernels' chunks) all give
    the plain logits."""
    cfg, tensors, folder, page = bc.case_folder(tmp_path, name, dtype=bc.stored_dtype(backend))
    n = 60 if name != "wide" else 130
    tokens = bc.clear_tokens(cfg, tensors, n, seed=1, dtype=backend[1])
    want = bc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = bc.make_replayer(folder, backend, 4 * 192, page)
    want.check(bc.feed(rp, "whole", tokens, [n]), "whole prompt")
    want.check(bc.feed(rp, "single", tokens, [] if n <= 60 else [n - 40]), "token by token")
    want.check(bc.feed(rp, "cut", tokens, [2, 3, 2, 7, 16, 2, 5, 9, 2]), "portions")
    want.check(bc.feed(rp, "cut2", tokens, [page + 1, 2 * page - 1, 2, 2, 17]), "portions across pages")
    if n > 100:
        want.check(bc.feed(rp, "cut3", tokens, [15, 2, 16, 17, 2, 63]), "portions at the edges of the kernels' chunks")
    assert rp.engine.cache.n_live() == 0


@pytest.mark.parametrize("backend", BACKENDS)
def test_batches_of_unequal_requests(tmp_path, backend):
    """Four live requests of different lengths, portions beside single tokens, in a pool so small
    that pages and state slots are used again: every request's logits are those it gets alone."""
    cfg, tensors, folder, page = bc.case_folder(tmp_path, "mixed", dtype=bc.stored_dtype(backend))
    lengths = [50, 9, 34, 1, 40, 2, 60]
    reqs = {f"r{i}": bc.clear_tokens(cfg, tensors, n, seed=10 + i, dtype=backend[1]) for i, n in enumerate(lengths)}
    want = {rid: bc.plain_logits(cfg, tensors, toks, backend[1]) for rid, toks in reqs.items()}
    rp = bc.make_replayer(folder, backend, 4 * 64, page, max_num_seqs=4)
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
def test_long_decoding_and_a_slot_used_again(tmp_path, backend):
    """A short prompt and 180 tokens decoded one by one (recorded steps on the GPU), then another
    request in the same state slot and pages: its first tokens must not feel the matrices, the
    convolutions' inputs and the last token that the first one left behind."""
    cfg, tensors, folder, page = bc.case_folder(tmp_path, "awkward", dtype=bc.stored_dtype(backend))
    tokens = bc.clear_tokens(cfg, tensors, 185, seed=3, dtype=backend[1])
    rp = bc.make_replayer(folder, backend, 192, page, max_num_seqs=1)
    bc.plain_logits(cfg, tensors, tokens, backend[1]).check(bc.feed(rp, "long", tokens, [5]), "long decoding")
    again = bc.clear_tokens(cfg, tensors, 20, seed=4, dtype=backend[1])
    bc.plain_logits(cfg, tensors, again, backend[1]).check(bc.feed(rp, "again", again, [1, 1, 3]), "the slot's next request")
    rp.engine.cache.check_invariants()


def test_layers_of_experts_as_one_matrix(tmp_path):
    """The form a decode batch takes on the GPU (every expert's [gate; up] as one matrix, zeros where a
    token did not choose an expert), forced for every step over the kernels' twins: the same logits."""
    from torch_ops import TorchOps
    from torchllms_b200.engine.replay import Replayer
    cfg, tensors, folder, page = bc.case_folder(tmp_path, "mixed")
    tokens = bc.clear_tokens(cfg, tensors, 40, seed=2, dtype="float32")
    ops = TorchOps()
    ops.dense_experts = True
    rp = Replayer(folder, "float32", 256, page_size=page, device="cpu", ops=ops, max_num_seqs=2)
    bc.plain_logits(cfg, tensors, tokens, "float32").check(bc.feed(rp, "a", tokens, [17, 2]), "all experts as one matrix")


# ---------------------------------------------------------------- one mechanism at a time

ALONE = {
    "left": dict(left=bc.attention(scaling=bc.ramp()), right_scale=0.0),
    "left-one-tap-whole-rotation": dict(left=bc.attention(heads=2, kv_heads=2, dim=8, vdim=8, conv=1, rot_dims=8, base=7.0), right_scale=0.0),
    "left-five-taps-no-rotation": dict(left=bc.attention(heads=2, kv_heads=1, dim=5, vdim=3, conv=5, rot_dims=0), right_scale=0.0),
    "left-eight-taps": dict(left=bc.attention(heads=1, kv_heads=1, dim=12, vdim=16, conv=8, rot_dims=8), right_scale=0.0),
    "right": dict(right=bc.delta(), left_scale=0.0),
    "right-one-tap": dict(right=bc.delta(heads=1, kv_heads=1, dim=4, vdim=4, conv=1), left_scale=0.0, ranks=(8, 1)),
    "right-six-taps-odd": dict(right=bc.delta(heads=3, kv_heads=1, dim=5, vdim=9, conv=6), left_scale=0.0, ranks=(2, 7)),
    "right-large-keys": dict(right=bc.delta(heads=2, kv_heads=2, dim=136, vdim=12, conv=2), left_scale=0.0, ranks=(16, 16)),
}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("kind", list(ALONE))
def test_each_mixer_alone(tmp_path, backend, kind):
    """One layer without a feed-forward and with one of its two mixers switched off by its scale."""
    cfg = bc.config([bc.layer(**ALONE[kind])], width=40, vocab=53)
    dtype = bc.stored_dtype(backend)
    tensors = bc.stored(bc.tensors_for(cfg, seed=len(kind), sharp=2.0 if backend[1] == "float32" else 1.0), dtype)
    tokens = bc.tokens_for(cfg, 70, seed=5)
    want = bc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = bc.make_replayer(bc.write_folder(tmp_path, kind, cfg, tensors, dtype), backend, 256, 8)
    want.check(bc.feed(rp, "p", tokens, [70]), "prompt")
    want.check(bc.feed(rp, "d", tokens, [3]), "decoded")
    want.check(bc.feed(rp, "c", tokens, [2, 2, 17, 2, 9, 16, 2]), "portions")


@pytest.mark.parametrize("backend", BACKENDS)
def test_a_far_key_at_a_pages_border(tmp_path, backend):
    """A key hundreds of places back, at a page's last and first place and at the sequence's start, that one query must
    find among all the others, in a prompt, in portions and when the query is decoded alone.  The test first proves on
    the plain implementation that losing that key moves the query's logits."""
    page, n, dk, rot = 8, 300, 12, 4
    cfg = bc.config([bc.layer(bc.attention(heads=2, kv_heads=1, dim=dk, vdim=8, conv=3, rot_dims=rot, scale=1.0), right_scale=0.1)],
                    width=32, vocab=400)
    dtype = bc.stored_dtype(backend)
    tokens = [int(x) for x in np.random.default_rng(5).permutation(400)[:n]]
    query_at = n - 3
    for key_at in (0, page * 3 - 1, page * 4):
        t = bc.tensors_for(cfg, seed=11)
        # coordinates 0 and 1 of the stream mark the key's and the query's token; the unrotated coordinate `rot` of a head
        # reads the first in k and the second in q, and the convolutions look at the current token alone there
        t["embed"][:, :2], t["bigram"] = 0.0, 0.1 * t["bigram"]
        t["bigram"][:, :2] = 0.0
        t["embed"][tokens[key_at], 0], t["embed"][tokens[query_at], 1] = 12.0, 12.0
        t["l0.norm1"][:2] = 1.0
        for name, heads, mark in (("q", 2, 1), ("k", 1, 0)):
            w, taps = t[f"l0.mix.left.{name}"], t[f"l0.mix.left.{name}.conv"]
            w[:, :2] = 0.0
            for h in range(heads):
                w[h * dk + rot] = 0.0
                w[h * dk + rot, mark] = 1.5
                taps[h * dk + rot] = torch.tensor([0.0, 0.0, 1.0])
        t = bc.stored(t, dtype)
        exact = plain.forward(cfg, t, tokens)
        lost = plain.forward(cfg, t, tokens[:key_at] + [tokens[key_at + 1]] + tokens[key_at + 1:])
        assert (exact[query_at] - lost[query_at]).abs().max() > 0.3, "the marked key does not matter: the test would say nothing"
        want = bc.plain_logits(cfg, t, tokens, backend[1])
        rp = bc.make_replayer(bc.write_folder(tmp_path, f"far{key_at}", cfg, t, dtype), backend, 2 * 320, page, max_num_seqs=2)
        want.check(bc.feed(rp, "p", tokens, [n]), "prompt")
        want.check(bc.feed(rp, "c", tokens, [key_at + 1, 2, 100, n - key_at - 103 - 8]), "portions, the query decoded alone")


@pytest.mark.parametrize("backend", BACKENDS)
def test_a_state_that_remembers_the_first_token(tmp_path, backend):
    """A matrix state that hardly forgets keeps its first token for hundreds of steps: the last logits
    depend on token 0 (proved on the plain implementation), so a state that is lost, zeroed or
    mixed up at the start of a portion or between steps shows."""
    dtype = bc.stored_dtype(backend)
    cfg = bc.config([bc.layer(right=bc.delta(heads=2, kv_heads=1, dim=64, vdim=12, conv=2), left_scale=0.0)], width=32, vocab=50, buckets=11)
    tensors = bc.tensors_for(cfg, seed=2)
    tensors["l0.mix.right.A_log"].fill_(-9.0)          # decays of all but one
    tensors["l0.mix.right.b"] = 0.05 * tensors["l0.mix.right.b"]
    tensors = bc.stored(tensors, dtype)
    n, marked = 160, cfg["vocab"] - 1
    tokens = [marked] + np.random.default_rng(5).integers(0, marked, size=n - 1).tolist()
    want = bc.plain_logits(cfg, tensors, tokens, backend[1])
    other = [0] + tokens[1:]
    assert np.abs(bc.plain_logits(cfg, tensors, other, backend[1]).logits[n - 1] - want.logits[n - 1]).max() > 0.03, \
        "the test's inputs do not show the first token at the end"
    rp = bc.make_replayer(bc.write_folder(tmp_path, "memory", cfg, tensors, dtype), backend, 512, 16)
    want.check(bc.feed(rp, "p", tokens, [n]), "prompt")
    want.check(bc.feed(rp, "d", tokens, [1]), "decoded from the second token on")
    want.check(bc.feed(rp, "c", tokens, [15, 2, 16, 17, 64, 2]), "portions around the chunk size")


@pytest.mark.parametrize("backend", BACKENDS)
def test_layers_that_share_weights_have_states_of_their_own(tmp_path, backend):
    """A layer that uses another's weights gives what a layer with equal tensors of its own gives; and the same
    tensors are not stored twice."""
    from torchllms_b200.engine.loading import load_model
    from torch_ops import TorchOps
    own = [bc.layer(), bc.layer(bc.attention(heads=2, kv_heads=1, conv=2), bc.delta(conv=3), mlp=bc.dense(40))]
    cfg = bc.config([own[0], own[1], bc.again(own, 0), bc.again(own, 1), bc.again(own, 0)], width=32, vocab=40)
    dtype = bc.stored_dtype(backend)
    tensors = bc.stored(bc.tensors_for(cfg, seed=6), dtype)
    full = bc.config([own[0], own[1], own[0], own[1], own[0]], width=32, vocab=40)
    spread = dict(tensors)
    for i, j in ((2, 0), (3, 1), (4, 0)):
        spread.update({f"l{i}." + k[3:]: v for k, v in tensors.items() if k.startswith(f"l{j}.")})
    tokens = bc.tokens_for(cfg, 40, seed=1)
    assert torch.equal(plain.forward(cfg, tensors, tokens), plain.forward(full, spread, tokens))
    folder = bc.write_folder(tmp_path, "shared", cfg, tensors, dtype)
    want = bc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = bc.make_replayer(folder, backend, 128, 8, max_num_seqs=2)
    want.check(bc.feed(rp, "a", tokens, [17, 2, 3]), "shared weights")
    assert len(rp.engine.model.blocks) == 2 and rp.engine.cache.n_runs == 5
    _, _, model = load_model(folder, dtype="float32", device="cpu", ops=TorchOps())
    assert len(model.blocks) == 2 and len(model.run_needs()) == 5 and model.step_weight_bytes() > model.weight_bytes()


def _without(name: str, cfg, tensors, tokens, monkeypatch):
    """Plain logits with one mechanism left out."""
    cfg, tensors = copy.deepcopy(cfg), {k: v.clone() for k, v in tensors.items()}
    with monkeypatch.context() as mp:
        if name == "pair rows":
            tensors["bigram"].zero_()
        elif name == "the first token's row":
            tensors["bigram"][-1] = 0.0
        elif name == "attention convolutions" or name == "delta convolutions":
            side = "left" if name.startswith("attention") else "right"
            for k, v in tensors.items():
                if f".{side}." in k and k.endswith(".conv"):
                    v[:, :-1] = 0.0
        elif name == "silu":
            mp.setattr(plain, "silu", lambda z: z)
        elif name == "ramp":
            for l in cfg["layers"]:
                l["mixer"]["left"]["rot"].pop("scaling", None)
        elif name == "growth of the rotated part":
            real = plain.rotate_half
            mp.setattr(plain, "rotate_half", lambda x, rot: torch.cat(
                [real(x, rot)[..., :rot["dims"]] / (0.1 * np.log(rot["scaling"]["factor"]) + 1.0), x[..., rot["dims"]:]], -1))
        elif name == "decay per channel":
            real_decay = plain.decay_of
            mp.setattr(plain, "decay_of", lambda *a: real_decay(*a).mean(-1, keepdim=True).expand_as(real_decay(*a)))
        elif name == "decay":
            mp.setattr(plain, "decay_of", lambda h, W, p, c, r: torch.ones(h.shape[0], c["heads"], c["dim"], dtype=F64))
        elif name == "unit vectors":
            mp.setattr(plain, "unit", lambda x: x)
        elif name == "attention gate":
            tensors["l0.mix.left.g"].zero_()
        elif name == "delta gate":
            tensors["l0.mix.right.g2"].zero_()
        elif name == "scales":
            for l in cfg["layers"]:
                l["mixer"]["left_scale"] = l["mixer"]["right_scale"] = 1.0
        elif name == "residual multiplier":
            cfg["residual_mult"] = 1.0
        elif name == "output norms":
            tensors["l0.norm1b"] = torch.ones_like(tensors["l0.norm1b"])
            tensors["l0.norm2b"] = torch.ones_like(tensors["l0.norm2b"])
        elif name == "correction":
            tensors["l0.mlp.correction"].zero_()
        elif name == "groups":
            del cfg["layers"][0]["mlp"]["router"]["groups"]
        elif name == "renormalised weights":
            real_route = plain.route
            mp.setattr(plain, "route", lambda *a: (lambda c, w: (c, w / w.sum(-1, keepdim=True)))(*real_route(*a)))
        else:
            raise ValueError(name)
        return plain.forward(cfg, tensors, tokens)


@pytest.mark.parametrize("backend", BACKENDS)
def test_every_mechanism_shows(tmp_path, backend, monkeypatch):
    """A model in which leaving out any one mechanism moves the plain logits: the engine holds to the real ones,
    from a sequence's first token on."""
    cfg = bc.config([bc.layer(bc.attention(heads=2, kv_heads=1, dim=10, vdim=6, conv=3, rot_dims=8, base=40.0, scaling=bc.ramp(6.0, 20, 6.0, 0.6)),
                              bc.delta(heads=2, kv_heads=1, dim=8, vdim=6, conv=3), left_scale=1.5, right_scale=0.7,
                              mlp=bc.moe(6, 2, 16, groups=(3, 1)), ranks=(4, 3))], width=24, vocab=61, mult=0.5)
    dtype = bc.stored_dtype(backend)
    tensors = bc.tensors_for(cfg, seed=3)
    tensors["l0.mlp.correction"] = torch.tensor([-0.6, -0.9, -0.4, -0.7, -0.55, -0.5])       # choice scores below zero
    tensors = bc.stored(tensors, dtype)
    tokens = bc.clear_tokens(cfg, tensors, 40, seed=8, dtype=backend[1])
    exact = plain.forward(cfg, tensors, tokens)
    for name in ("pair rows", "the first token's row", "attention convolutions", "delta convolutions", "silu", "ramp",
                 "growth of the rotated part", "decay per channel", "decay", "unit vectors", "attention gate", "delta gate", "scales",
                 "residual multiplier", "output norms", "correction", "groups"):
        assert (_without(name, cfg, tensors, tokens, monkeypatch) - exact).abs().max() > 0.05, name
    # (the norm on a sublayer's output hides a common factor of the weights from the stream, but for its epsilon)
    assert (_without("renormalised weights", cfg, tensors, tokens, monkeypatch) - exact).abs().max() < 0.05
    want = bc.plain_logits(cfg, tensors, tokens, backend[1])
    rp = bc.make_replayer(bc.write_folder(tmp_path, "all", cfg, tensors, dtype), backend, 128, 4)
    want.check(bc.feed(rp, "p", tokens, [40]), "prompt")
    want.check(bc.feed(rp, "d", tokens, []), "token by token from the first")
    want.check(bc.feed(rp, "c", tokens, [1, 2, 3, 9]), "portions")


# ---------------------------------------------------------------- kernels against the plain functions

def _ops(backend):
    if backend[0] == "cpu":
        from torch_ops import TorchOps
        return TorchOps(), torch.device("cpu")
    from torchllms_b200.kernels import get_ops
    return get_ops(), torch.device("cuda")


def _dt(backend):
    return torch.bfloat16 if backend[1] == "bfloat16" else torch.float32


def _i32(xs, dev):
    return torch.tensor(xs, dtype=torch.int32, device=dev)


def _steps(lens, slots, fresh, dev):
    start = np.concatenate([[0], np.cumsum(lens)]).tolist()
    return (_i32(start, dev), _i32(slots, dev), _i32([int(f) for f in fresh], dev)), dict(n_seqs=len(lens), max_q_len=max(lens))


@pytest.mark.parametrize("backend", BACKENDS)
def test_embedding_of_pairs(backend):
    """Portions of several requests, fresh ones and ones that go on: the row of every pair, the last row at a request's
    start, products of token and multiplier beyond 32 bits, negative multipliers, and the last token left behind."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(1)
    for dim, vocab, buckets, mul_prev, mul_cur in ((8, 11, 7, 3, 5), (30, 90000, 13, 1 << 40, 987654321), (64, 50, 1, 2, 3), (20, 40, 9, -7, 4)):
        table, rows = (torch.randn(vocab, dim, generator=g).to(_dt(backend)) for vocab in (vocab, buckets + 1))
        lens, slots, fresh = [5, 1, 1, 3], [2, 0, 3, 1], [True, False, True, False]
        ids = torch.randint(0, vocab, (sum(lens),), generator=g)
        last = torch.tensor([[vocab - 1], [4], [6], [8]], dtype=torch.int32)
        want, at, after = [], 0, last.clone()
        for n, slot, f in zip(lens, slots, fresh):
            before = [] if f else [int(last[slot, 0])]
            toks = torch.tensor(before + ids[at:at + n].tolist())
            picked = plain.bigram_rows(toks, {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur})[len(before):]
            want.append(table[ids[at:at + n]].double() + rows[picked].double())
            after[slot, 0] = ids[at + n - 1]
            at += n
        seq = torch.repeat_interleave(torch.arange(4), torch.tensor(lens)).to(torch.int32).to(dev)
        (q_start, slot_t, fresh_t), _how = _steps(lens, slots, fresh, dev)
        held = last.to(dev)
        got = ops.embed_pairs(ids.to(torch.int32).to(dev), table.to(dev), rows.to(dev), held, seq, q_start, slot_t, fresh_t,
                              mul_prev=mul_prev, mul_cur=mul_cur)
        torch.testing.assert_close(got.cpu().double(), torch.cat(want), atol=1e-6, rtol=1e-6)
        assert torch.equal(held.cpu(), after)


def _convolved(x, w, before, lens, fresh):
    """Plain convolution of every request's portion (float64), and the inputs each leaves behind."""
    out, left, at, taps = [], [], 0, w.shape[1]
    for b, (n, f) in enumerate(zip(lens, fresh)):
        full = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F64) if f else before[b].double(), x[at:at + n].double()])
        out.append(plain.causal_conv(full, w.double())[taps - 1:])
        left.append(full[full.shape[0] - (taps - 1):])
        at += n
    return torch.cat(out), left


# portions: a long one, a decoded token that goes on from a state, a fresh short one, a short one that goes on
LENS, SLOTS, FRESH = [37, 1, 3, 2], [2, 0, 3, 1], [True, False, True, False]


@pytest.mark.parametrize("backend", BACKENDS)
def test_convolution_rotation_and_store(backend):
    """The kernel behind the input projection of an attention with short convolutions: several numbers of taps, sizes that are
    and are not multiples of four, rotations over a part of a head, all of it and none, a gate with a scale, rows that are
    a column range of wider ones, partial sums, steps of long and of short portions, states that are fields of wider rows."""
    from torchllms_b200.parts.rope import precise_rotary_table
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(3)
    dt = _dt(backend)
    page = 4
    for H, G, d, dv, rot, taps, extra in ((4, 2, 16, 24, 8, 3, 96), (3, 1, 10, 7, 6, 1, 21), (2, 2, 64, 128, 64, 4, 256), (5, 1, 9, 6, 0, 2, 0),
                                          (2, 1, 32, 8, 16, 8, 16), (1, 1, 12, 20, 12, 6, 20)):
        rotary = {"dims": rot, "base": 500.0, "scaling": bc.ramp(3.0, 50, 8.0, 1.0)}
        table = precise_rotary_table(max(rot, 2), 500.0, 1.0, 200, dev, ramp=rotary["scaling"] if rot else None)
        C, W = (H + G) * d + G * dv, (H + G) * d + G * dv + extra
        for lens, slots, fresh in ((LENS, SLOTS, FRESH), ([1, 1, 2, 1], SLOTS, FRESH), ([16, 5, 1, 9], SLOTS, FRESH)):
            T = sum(lens)
            for splits, off in ((1, 0), (1, 3), (2, 8)):
                wide = torch.randn(splits, T, W + 2 * off, generator=g).to(torch.float32 if splits > 1 else dt)
                x = wide.double().sum(0)[:, off:off + W]
                w = torch.randn(C, taps, generator=g)
                before = torch.randn(len(lens), max(taps - 1, 0), C, generator=g)
                state_all = torch.zeros(4, (taps - 1) * C + 8)
                field = lambda s: s[:, 4:4 + (taps - 1) * C].unflatten(1, (taps - 1, C)) if taps > 1 else None
                if taps > 1:
                    field(state_all)[:] = 9.0                  # left behind by earlier requests: fresh ones must not read it
                    for b, (slot, f) in enumerate(zip(slots, fresh)):
                        if not f:
                            field(state_all)[slot] = before[b]
                y, left = _convolved(x[:, :C], w, before, lens, fresh)
                pos = torch.cat([torch.arange(40 + 7 * b, 40 + 7 * b + n) for b, n in enumerate(lens)])
                q = y[:, :H * d].view(T, H, d)
                k = y[:, H * d:(H + G) * d].view(T, G, d)
                v = y[:, (H + G) * d:C].view(T, G, dv)
                if rot:
                    turn = lambda z: torch.stack([plain.rotate_half(z[t:t + 1].expand(int(p) + 1, -1, -1), rotary)[int(p)] for t, p in enumerate(pos)])
                    q, k = turn(q), turn(k)
                pages = -(-T // page) + 1
                sm = torch.randperm(pages * page, generator=g)[:T]
                kp = torch.full((pages, G, page, d), 7.0, dtype=dt, device=dev)
                vp = torch.full((pages, G, page, dv), 7.0, dtype=dt, device=dev)
                (q_start, slot_t, fresh_t), how = _steps(lens, slots, fresh, dev)
                held = state_all.to(dev)
                view = wide.to(dev)[..., off:off + W]
                got_q, gate = ops.conv_rope_store(view if splits > 1 else view[0], w.t().contiguous().to(dev), field(held), pos.to(torch.int32).to(dev), table, q_start,
                                                  slot_t, fresh_t, n_q_heads=H, n_k_heads=G, head_dim=d, v_head_dim=dv, rot_dims=rot,
                                                  n_extra=extra, k_pages=kp, v_pages=vp, slot_mapping=sm.to(torch.int32).to(dev),
                                                  page_size=page, out_dtype=dt, extra_scale=1.7, **how)
                tol = dict(atol=2e-4, rtol=2e-4) if dt == torch.float32 else dict(atol=2e-2, rtol=2e-2)
                torch.testing.assert_close(got_q.cpu().double(), q, **tol)
                torch.testing.assert_close(kp[sm // page, :, sm % page].cpu().double(), k, **tol)
                torch.testing.assert_close(vp[sm // page, :, sm % page].cpu().double(), v, **tol)
                if extra:
                    torch.testing.assert_close(gate.cpu().double(), 1.7 * torch.sigmoid(x[:, C:]), **tol)
                else:
                    assert gate is None
                if taps > 1:
                    for slot, rows in zip(slots, left):
                        torch.testing.assert_close(field(held)[slot].cpu().double(), rows, atol=1e-5, rtol=1e-5)
                assert torch.equal(held.cpu()[:, :4], state_all[:, :4]), "the state's neighbours changed"


@pytest.mark.parametrize("backend", BACKENDS)
def test_preparing_a_delta_rule(backend):
    """Convolution, silu, unit vectors, and the columns behind: numbers of taps, head sizes in and out of fours and beyond
    128, rows that are column ranges, partial sums, long and short portions."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(4)
    dt = _dt(backend)
    for heads, d, n_v, taps, n_small, n_low in ((2, 12, 80, 2, 4, 14), (1, 7, 33, 1, 3, 0), (3, 64, 256, 4, 8, 160), (2, 160, 36, 3, 2, 24), (1, 130, 10, 7, 1, 5)):
        n, W = heads * d, 2 * heads * d + n_v + n_small + n_low + 3
        C = 2 * n + n_v
        for lens, slots, fresh in ((LENS, SLOTS, FRESH), ([1, 1, 2, 1], SLOTS, FRESH)):
            T = sum(lens)
            for splits, off in ((1, 0), (1, 5), (3, 4)):
                wide = torch.randn(splits, T, W + off, generator=g).to(torch.float32 if splits > 1 else dt)
                x = wide.double().sum(0)[:, off:]
                w = torch.randn(C, taps, generator=g)
                before = torch.randn(len(lens), max(taps - 1, 0), C, generator=g)
                state = torch.full((4, max(taps - 1, 1), C), 9.0)
                for b, (slot, f) in enumerate(zip(slots, fresh)):
                    if taps > 1 and not f:
                        state[slot] = before[b]
                y, left = _convolved(x[:, :C], w, before, lens, fresh)
                y = plain.silu(y)
                q = (plain.unit(y[:, :n].view(T, heads, d)) * 0.3).flatten(1)
                k = plain.unit(y[:, n:2 * n].view(T, heads, d)).flatten(1)
                (q_start, slot_t, fresh_t), how = _steps(lens, slots, fresh, dev)
                held = state.to(dev) if taps > 1 else None
                view = wide.to(dev)[..., off:]
                pad = -(-n_low // 8) * 8
                got = ops.delta_prep(view if splits > 1 else view[0], w.t().contiguous().to(dev), held, q_start, slot_t, fresh_t, n_qk_heads=heads, head_dim=d, n_v=n_v,
                                     n_small=n_small, n_low=n_low, low_pad=pad, q_scale=0.3, unit_eps=1e-6, out_dtype=dt, **how)
                tol = dict(atol=2e-5, rtol=2e-5) if dt == torch.float32 else dict(atol=2e-2, rtol=2e-2)
                torch.testing.assert_close(got[0].cpu().double(), q, atol=2e-5, rtol=1e-4)
                torch.testing.assert_close(got[1].cpu().double(), k, atol=2e-5, rtol=1e-4)
                torch.testing.assert_close(got[2].cpu().double(), y[:, 2 * n:], **tol)
                torch.testing.assert_close(got[3].cpu().double(), x[:, C:C + n_small], **tol)
                if n_low:
                    torch.testing.assert_close(got[4].cpu().double()[:, :n_low], x[:, C + n_small:C + n_small + n_low], **tol)
                    assert not got[4][:, n_low:].any()
                else:
                    assert got[4] is None
                if taps > 1:
                    for slot, rows in zip(slots, left):
                        torch.testing.assert_close(held[slot].cpu().double(), rows, atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("backend", BACKENDS)
def test_delta_rule_with_a_decay_per_channel(backend):
    """The recurrence over long portions (decays from a kernel of their own) and short ones (worked out where they are used),
    shared heads of q and k, key sizes up to 256 in and out of fours, decays close to one and to zero, states that go on."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(5)
    dt = _dt(backend)
    for H, G, d, dv in ((3, 1, 10, 6), (4, 2, 32, 64), (2, 2, 96, 40), (2, 1, 64, 17), (1, 1, 130, 33), (2, 1, 256, 20)):
        for lens in (LENS, [1, 1, 4, 2]):
            T = sum(lens)
            q = torch.nn.functional.normalize(torch.randn(T, G, d, generator=g), dim=-1) * d ** -0.5
            k = torch.nn.functional.normalize(torch.randn(T, G, d, generator=g), dim=-1)
            wide = torch.randn(T, H * dv + H + H * d + 5, generator=g).to(dt)
            v, beta = wide[:, 1:1 + H * dv], wide[:, 1 + H * dv:1 + H * dv + H]
            z = wide[:, 2 + H * dv + H:2 + H * dv + H + H * d]
            rate, bias = torch.rand(H, generator=g) + 0.1, 4.0 * torch.randn(H * d, generator=g)
            decay = torch.exp(-rate.double()[:, None] * torch.nn.functional.softplus(z.double() + bias.double()).view(T, H, d))
            state = torch.full((4, H, dv, d), 5.0)
            held = {slot: torch.randn(H, d, dv, generator=g) for slot, f in zip(SLOTS, FRESH) if not f}
            for slot, S in held.items():
                state[slot] = S.transpose(1, 2)
            want, new, at = [], {}, 0
            for n, slot, f in zip(lens, SLOTS, FRESH):
                S = torch.zeros(H, d, dv, dtype=F64) if f else held[slot].double()
                for t in range(at, at + n):
                    o = torch.zeros(H, dv, dtype=F64)
                    for a in range(H):
                        kt, qt = k[t, a // (H // G)].double(), q[t, a // (H // G)].double()
                        M = decay[t, a][:, None] * S[a]
                        u = torch.sigmoid(beta[t, a].double()) * (v[t, a * dv:(a + 1) * dv].double() - M.T @ kt)
                        M = M + torch.outer(kt, u)
                        S[a] = M
                        o[a] = M.T @ qt
                    want.append(o.flatten())
                new[slot] = S
                at += n
            (q_start, slot_t, fresh_t), how = _steps(lens, SLOTS, FRESH, dev)
            sd, wd = state.to(dev), wide.to(dev)
            got = ops.linear_recurrence(q.flatten(1).to(dev), k.flatten(1).to(dev), wd[:, 1:1 + H * dv], sd, q_start, slot_t, fresh_t,
                                        beta_logits=wd[:, 1 + H * dv:1 + H * dv + H], decay_logits=wd[:, 2 + H * dv + H:2 + H * dv + H + H * d],
                                        decay_rate=rate.to(dev), decay_bias=bias.to(dev), **how)
            want = torch.stack(want)
            torch.testing.assert_close(got.cpu().double(), want, atol=2e-5 * float(want.abs().max()), rtol=1e-4)
            for slot, S in new.items():
                torch.testing.assert_close(sd[slot].cpu().double(), S.transpose(1, 2), atol=2e-5 * float(S.abs().max()), rtol=1e-4)
            # a plain decay per channel and its own equations agree with the function of the plain implementation
            first = lens[0]
            of_plain = plain.channel_delta(q[:first].double(), k[:first].double(), v[:first].double().view(first, H, dv),
                                           torch.sigmoid(beta[:first].double()), decay[:first]).flatten(1)
            torch.testing.assert_close(of_plain, want[:first], atol=1e-9, rtol=1e-9)


@pytest.mark.parametrize("backend", BACKENDS)
def test_results_that_are_columns_of_wider_rows(backend):
    """The head norm with a sigmoid gate, and attention with a gate in one key split and in several, writing into a column
    range of wider rows: the same numbers as into a tensor of their own, and nothing beside the range."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(6)
    dt = _dt(backend)
    tol = dict(atol=2e-5, rtol=2e-5) if dt == torch.float32 else dict(atol=2e-2, rtol=2e-2)
    for T, H, d in ((1, 3, 10), (9, 4, 32), (70, 2, 96)):
        o, z, w = torch.randn(T, H * d, generator=g), torch.randn(T, H * d + 3, generator=g).to(dt), torch.randn(d, generator=g)
        want = (plain.rms(o.double().view(T, H, d), 1e-5) * w.double()).flatten(1) * torch.sigmoid(z.double()[:, 3:])
        rows = torch.full((T, H * d + 9), 3.0, dtype=dt, device=dev)
        ops.head_norm_gate(o.to(dev), z.to(dev)[:, 3:], w.to(dev), 1e-5, head_dim=d, out_dtype=dt, activation="sigmoid", out=rows[:, 5:5 + H * d])
        torch.testing.assert_close(rows[:, 5:5 + H * d].cpu().double(), want, **tol)
        assert (rows[:, :5] == 3.0).all() and (rows[:, 5 + H * d:] == 3.0).all()
    page = 8
    for H, G, d, dv, width in ((4, 2, 16, 24, 4 * 24 + 10), (2, 1, 9, 7, 2 * 7 + 3), (6, 2, 40, 80, 6 * 80 + 64)):
        for lens, total in (([1, 1], [700, 90]), ([40, 3], [60, 200])):
            T = sum(lens)
            n_pages = sum(-(-n // page) for n in total)
            kp = torch.randn(n_pages, G, page, d, generator=g).to(dt).to(dev)
            vp = torch.randn(n_pages, G, page, dv, generator=g).to(dt).to(dev)
            table = torch.full((2, -(-max(total) // page)), -1, dtype=torch.int32)
            at = 0
            for b, n in enumerate(total):
                k = -(-n // page)
                table[b, :k] = torch.arange(at, at + k)
                at += k
            q = torch.randn(T, H, d, generator=g).to(dt).to(dev)
            gate = torch.rand(T, H * dv, generator=g).to(dt).to(dev)
            (q_start, _s, _f), how = _steps(lens, [0, 1], [0, 0], dev)
            run = lambda out: ops.paged_attention(q, kp, vp, table.to(dev), q_start, _i32(total, dev), max_kv_len=max(total), scale=0.3, window=None,
                                                  page_size=page, gate=gate, **how, **({} if out is None else dict(out=out)))
            alone = run(None).flatten(1)
            rows = torch.full((T, width), 3.0, dtype=dt, device=dev)
            run(rows[:, :H * dv].unflatten(1, (H, dv)))
            torch.testing.assert_close(rows[:, :H * dv], alone, **tol)
            assert (rows[:, H * dv:] == 3.0).all()


@pytest.mark.parametrize("backend", BACKENDS)
def test_router_with_groups_scored_by_their_best(backend):
    """Choice scores below zero, groups scored by their best choice score, weights as the softmax gives them."""
    ops, dev = _ops(backend)
    g = torch.Generator().manual_seed(7)
    for E, top, count, keep in ((12, 3, 2, 1), (8, 2, 4, 2), (9, 3, 3, 3), (6, 1, 6, 1), (10, 4, 1, 1)):
        for T in (5, 90):
            x = torch.randn(T, 24, generator=g).to(_dt(backend))
            w, c = torch.randn(E, 24, generator=g) * 0.3, -1.0 + 0.5 * torch.randn(E, generator=g)
            router = {"top": top, "groups": {"count": count, "keep": keep}} if count > 1 else {"top": top}
            margins: list = []
            chosen, weights = plain.route(x.double() @ w.double().T, c.double(), router, margins)
            got_c, got_w, _ = ops.moe_route(x.to(dev), w.to(dev), c.to(dev), n_experts=E, top=top, scale=1.0, renormalize=False, shared_gate=False,
                                            n_groups=count, keep_groups=keep, group_score_top=1)
            clear = margins[0] > 1e-4
            assert clear.float().mean() > 0.9
            want, order = chosen.sort(-1)
            have, places = got_c.cpu().long().sort(-1)
            assert torch.equal(have[clear], want[clear])
            torch.testing.assert_close(got_w.cpu().double().gather(1, places)[clear], weights.gather(1, order)[clear], atol=2e-5, rtol=2e-4)


def test_frequencies_along_a_ramp():
    """The table against the plain frequencies: pairs below the ramp, on it and beyond, ramps that end outside the pairs or
    have no length, far positions, and no rescaling at all."""
    from torchllms_b200.parts.rope import precise_rotary_table
    for dims, base, s in ((32, 10000.0, bc.ramp(8.0, 512, 32.0, 1.0)), (12, 50.0, bc.ramp(2.0, 64, 4.0, 2.0)), (8, 3.0, bc.ramp(4.0, 10, 50.0, 0.01)),
                          (16, 1e6, bc.ramp(5.0, 4096, 4096.0, 4095.0)), (6, 100.0, None)):
        rot = {"dims": dims, "base": base, **({} if s is None else {"scaling": s})}
        f = torch.tensor(plain.frequencies(rot), dtype=F64)
        grow = 1.0 if s is None else 0.1 * np.log(s["factor"]) + 1.0
        table = precise_rotary_table(dims, base, 1.0, 5000, ramp=s)
        for p in (0, 1, 17, 4999):
            torch.testing.assert_close(table[p].double(), grow * torch.stack([torch.cos(p * f), torch.sin(p * f)], -1), atol=2e-7, rtol=2e-7)


def test_configuration_and_names(tmp_path):
    """config.json is read key by key, written back as it was read, and refused with the key's name
    when something is off; the checkpoint's names reach the parts, and a tensor too many or too few
    is reported by name."""
    from torchllms_b200.config.model_config import ConfigError
    from torchllms_b200.config.registry import load_config
    from torchllms_b200.engine.loading import load_model
    from torch_ops import TorchOps
    cfg, tensors, folder, _page = bc.case_folder(tmp_path, "mixed")
    arch, parsed = load_config(folder)
    assert arch.name == "Bomotar" and parsed.to_hf() == bc.clean(cfg)
    assert parsed.layers[0].mixer.left.scaling.original == 64 and parsed.layers[2].weights_of == 0 and parsed.owners() == [0, 1]
    assert parsed.layers[0].mlp.keep_groups == 2 and parsed.mul_prev == 17
    _arch, odd = load_config(bc.case_folder(tmp_path, "awkward")[2])
    assert [odd.owner(i) for i in range(4)] == [2, 1, 2, 2] and odd.layers[1].mlp.groups == 1 and odd.layers[2].mixer.left.scaling is None
    for n, (path, value, word) in enumerate((
            (("layers", 0, "mixer", "left", "kv_heads"), 3, "kv_heads"), (("layers", 1, "type"), "other", "other"),
            (("layers", 0, "mixer", "right", "conv"), 0, "conv"), (("layers", 0, "mixer", "left", "rot", "dims"), 5, "rot.dims"),
            (("layers", 0, "mlp", "router", "top"), 9, "top"), (("layers", 0, "mlp", "router", "groups", "count"), 3, "groups"),
            (("layers", 2, "weights_of"), 1, "weights_of"), (("layers", 2, "weights_of"), 2, "weights_of"), (("layers", 2, "weights_of"), 4, "weights_of"),
            (("embedding", "bigram", "buckets"), 0, "buckets"), (("residual_mult",), None, "residual_mult"),
            (("layers", 0, "mixer", "left", "rot", "scaling", "slow"), 0.0, "scaling"))):
        bad = copy.deepcopy(bc.clean(cfg))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        sub = tmp_path / f"bad_{n}"
        sub.mkdir()
        (sub / "config.json").write_text(json.dumps(bad))
        with pytest.raises(ConfigError, match=word):
            load_config(sub)
    _, _, model = load_model(folder, dtype="float32", device="cpu", ops=TorchOps())
    assert model.blocks[0].mixer.members[0][1].n_heads == 4 and model.blocks[1].mixer.members[1][1].taps == 3
    lost = dict(tensors)
    del lost["l1.mix.left.k.conv"]
    lost["l0.mix.extra"] = torch.zeros(2)
    with pytest.raises(Exception, match="l1.mix.left.k_?.*conv|l0.mix.extra"):
        load_model(bc.write_folder(tmp_path, "lost", cfg, lost), dtype="float32", device="cpu", ops=TorchOps())
    uneven = dict(tensors)
    uneven["l0.mix.right.a2"] = torch.zeros(tensors["l0.mix.right.a2"].shape[0], 4)
    with pytest.raises(ValueError, match="low-rank"):
        load_model(bc.write_folder(tmp_path, "uneven", cfg, uneven), dtype="float32", device="cpu", ops=TorchOps())


@pytest.mark.parametrize("backend", BACKENDS)
def test_greedy_generation_through_the_scheduler(tmp_path, backend):
    """``LLM.generate`` (scheduler, sampler, look-ahead) against a plain greedy loop."""
    from torchllms_b200.inference import LLM
    cfg, tensors, folder, page = bc.case_folder(tmp_path, "mixed", dtype=bc.stored_dtype(backend))
    kw = {}
    if backend[0] == "cpu":
        from torch_ops import TorchOps
        kw = dict(ops=TorchOps())
    llm = LLM(folder, max_len=128, max_bsz=3, device=backend[0], precision=backend[1], page_size=page,
              max_num_batched_tokens=24, **kw)
    prompts = [bc.clear_tokens(cfg, tensors, n, seed=20 + n, dtype=backend[1]) for n in (3, 30, 11, 1)]
    results = llm.generate(prompt_token_ids=prompts, temperature=0.0, max_new_tokens=12, disable_tqdm=True)
    margin = 1e-3 if backend[1] == "float32" else 0.1
    router_margin = 1e-4 if backend[1] == "float32" else 0.03
    compared = 0
    for prompt, r in zip(prompts, results):
        seq = list(prompt)
        for _ in range(12):
            margins: list = []
            logits = plain.forward(cfg, tensors, seq, margins_out=margins)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) < margin or min(float(m.min()) for m in margins) < router_margin:
                break                         # a near tie may fall either way: stop comparing this request
            seq.append(int(torch.argmax(logits)))
        made = seq[len(prompt):]
        compared += len(made)
        assert r.error is None and len(r.token_ids) == 12 and r.token_ids[:len(made)] == made
    assert compared >= (40 if backend[1] == "float32" else 1)


def test_random_weights_mode_writes_a_folder_that_loads(tmp_path):
    """The framework's random-weights mode for this architecture: a folder under the checkpoint's
    names that loads like any other, and the same model built without a file."""
    from torchllms_b200.config.registry import load_config
    from torchllms_b200.engine.loading import load_model, random_model
    from torchllms_b200.weights.random_init import write_random_model
    from torchllms_b200.weights.safetensors_io import TensorSource
    from torch_ops import TorchOps
    _cfg, _tensors, folder, _page = bc.case_folder(tmp_path, "mixed")
    _arch, parsed = load_config(folder)
    out = write_random_model(tmp_path / "random", parsed, seed=3)
    names = set(TensorSource(out).names())
    assert {"embed", "bigram", "head", "final.norm", "l0.mix.left.q.conv", "l1.mix.right.a2", "l0.mlp.e7.gate", "l1.norm2b"} <= names
    assert not any(n.startswith(("l2.", "l3.")) for n in names)
    _, _, from_file = load_model(out, dtype="float32", device="cpu", ops=TorchOps())
    _, _, direct = random_model(parsed, 3, dtype="float32", device="cpu", ops=TorchOps())
    assert torch.equal(from_file.pair_rows, direct.pair_rows)
    assert torch.equal(from_file.blocks[1].mixer.w_in, direct.blocks[1].mixer.w_in)
