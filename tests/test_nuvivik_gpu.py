"""Nuvivik on the GPU against the plain oracle (tests/plain/nuvivik_plain.py): every mechanism alone, whole prompts,
decoding through the cache, prompts in pieces, batches against each request alone, reuse of slots and pages, the edges of
windows and pages, the first tokens, far keys, long decoding, other sizes, and generation through the engine, the replay
program and the command line."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from nuvivik_cases import CASES, assert_rows, attention, latent, make_folder, model, moe, oracle_view, row_errors, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
SMALL = ["A", "B", "C", "D"]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("nuvivik")
    return {k: make_folder(base, raw, seed, k) for k, (raw, seed) in CASES.items()}


def _runner(folder, dtype, **kw):
    from hos_b200.engine import Runner
    kw.setdefault("max_tokens", 4096)
    kw.setdefault("max_seq_len", 1024)
    return Runner.from_folder(folder, dtype=dtype, **kw)


def _oracle(folder, seqs):
    from plain import nuvivik_plain as P
    cfg, w = oracle_view(folder)
    return [P.forward(cfg, w, s) for s in seqs]


def _resized(cfg, d):
    """An edit that makes every window d keys longer, or None if a window would be empty or there is none."""
    masks = [l["mixer"]["mask"]["size"] for l in cfg["layers"] if l["mixer"].get("mask")]
    if not masks:
        return None

    def edit(i, m):
        return dict(m, mask={"size": m["mask"]["size"] + d}) if m.get("mask") and m["mask"]["size"] + d > 0 else m
    return edit


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", SMALL)
def test_whole_prompts_of_unequal_lengths(folders, case, dtype):
    vocab = CASES[case][0]["vocab"]
    seqs = [tokens(i, n, vocab) for i, n in enumerate((1, 2, 37, 150))]      # 150: beyond two pages and every window
    want = _oracle(folders[case], seqs)
    r = _runner(folders[case], dtype)
    slots = r.admit(len(seqs))
    got = r.step(slots, seqs, [list(range(len(s))) for s in seqs]).cpu()
    assert_rows(got, torch.cat(want), dtype, f"case {case}")
    for s in slots:
        r.release(s)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", SMALL)
def test_a_prompt_then_token_by_token(folders, case, dtype):
    """Two requests decoded side by side through the replayed single-token step, across page borders (64, 128) and every
    window's edge, with rings of pages that are written round; the shorter one leaves first.  The longer one is decoded for
    141 steps, so every window passes wholly over decoded tokens."""
    vocab = CASES[case][0]["vocab"]
    seqs = [tokens(20, 150, vocab), tokens(21, 90, vocab)]
    plens = [9, 61]
    want = _oracle(folders[case], seqs)
    r = _runner(folders[case], dtype, chunk_tokens=1)
    slots = r.admit(2)
    first = r.step(slots, [s[:n] for s, n in zip(seqs, plens)]).cpu()
    got = [[first[0:1]], [first[1:2]]]
    pos, live = list(plens), [0, 1]
    while live:
        out = r.step([slots[i] for i in live], [[seqs[i][pos[i]]] for i in live]).cpu()
        for j, i in enumerate(live):
            got[i].append(out[j:j + 1])
            pos[i] += 1
        for i in [i for i in live if pos[i] == len(seqs[i])]:
            r.release(slots[i])
        live = [i for i in live if pos[i] < len(seqs[i])]
    for i in range(2):
        assert_rows(torch.cat(got[i]), want[i][plens[i] - 1:], dtype, f"case {case} request {i}")
    r.cache.check()


@pytest.mark.parametrize("case, dtype, room", [("A", "float32", 20), ("A", "bfloat16", 2048), ("B", "float32", 7), ("C", "float32", 2048),
                                               ("C", "bfloat16", 20), ("D", "bfloat16", 64)])
def test_a_prompt_in_pieces_of_many_sizes(folders, case, dtype, room):
    """Pieces down to two tokens and one, pieces that end on a page's border and one past it, in rings that hold little
    more than the window (a piece then runs in several passes) and in rings that hold much more."""
    vocab = CASES[case][0]["vocab"]
    seq = tokens(30, 230, vocab)
    want = _oracle(folders[case], [seq])[0]
    r = _runner(folders[case], dtype, chunk_tokens=room)
    (slot,) = r.admit(1)
    at, got = 0, []
    for k in [2, 3, 59, 1, 65, 7, 2, 40, 1, 1, 30, 19]:
        piece = seq[at:at + k]
        got.append(r.step([slot], [piece], [list(range(len(piece)))]).cpu())
        at += len(piece)
    assert at == len(seq)
    assert_rows(torch.cat(got), want, dtype, f"case {case}")
    r.release(slot)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["A", "C"])
def test_a_batch_gives_what_each_request_gives_alone(folders, case, dtype):
    """Also a step in which one request starts while others go on by one token and by several."""
    vocab = CASES[case][0]["vocab"]
    seqs = [tokens(40 + i, n, vocab) for i, n in enumerate((75, 3, 130))]
    r = _runner(folders[case], dtype)
    alone = []
    for s in seqs:
        (slot,) = r.admit(1)
        alone.append(r.step([slot], [s], [list(range(len(s)))]).cpu())
        r.release(slot)
    slots = r.admit(3)
    both = r.step(slots, seqs, [list(range(len(s))) for s in seqs]).cpu()
    for s in slots:
        r.release(s)
    tol = 2e-5 if dtype == "float32" else 4e-2
    assert float(row_errors(both, torch.cat(alone)).max()) <= tol
    slots = r.admit(2)
    r.step(slots, [seqs[0][:74], seqs[2][:100]])
    (late,) = r.admit(1)
    mixed = r.step([late, slots[1], slots[0]], [seqs[1], seqs[2][100:109], seqs[0][74:75]],
                   [[0, 1, 2], list(range(9)), [0]]).cpu()
    ref = torch.cat([alone[1], alone[2][100:109], alone[0][74:75]])
    assert float(row_errors(mixed, ref).max()) <= tol
    r.cache.check()


def test_slots_and_pages_that_are_freed_are_used_again(folders):
    """What a freed slot's pages still hold must never be read."""
    vocab = CASES["A"][0]["vocab"]
    first, second = tokens(50, 140, vocab), tokens(51, 100, vocab)
    want = _oracle(folders["A"], [second])[0]
    r = _runner(folders["A"], "float32", max_tokens=256)       # four pages: the second request must reuse them
    (slot,) = r.admit(1)
    r.step([slot], [first[:130]])
    for t in first[130:]:
        r.step([slot], [[t]])
    r.release(slot)
    for g in r.cache.groups:
        for t in g.k + g.v:
            if t is not None:            # a keys-only group has no values
                t.fill_(1e4)
    (again,) = r.admit(1)
    assert again == slot
    got = [r.step([again], [second[:70]], [list(range(70))]).cpu()]
    for t in second[70:]:
        got.append(r.step([again], [[t]]).cpu())
    assert_rows(torch.cat(got), want, "float32", "second request in a used slot")
    r.release(again)
    (again,) = r.admit(1)                # and one that starts with single tokens
    got = [r.step([again], [[t]]).cpu() for t in second[:12]]
    assert_rows(torch.cat(got), want[:12], "float32", "token by token from the first in a used slot")
    r.release(again)
    r.cache.check()


@pytest.mark.parametrize("case", SMALL)
def test_the_edges_of_every_window_in_prompts_and_in_decoding(folders, case):
    """The oracle with every window one key longer or shorter is far from the oracle itself (so an edge that is off by one
    cannot pass), and the library agrees with the oracle at every position, whether the token comes in a prompt or alone."""
    from plain import nuvivik_plain as P
    cfg, w = oracle_view(folders[case])
    seq = tokens(60, 160, cfg["vocab"])
    want = P.forward(cfg, w, seq)
    for d in (1, -1):
        edit = _resized(cfg, d)
        # one key more or fewer among up to 100: at least ten times what the 32-bit comparison below allows
        assert float(row_errors(P.forward(cfg, w, seq, edit=edit)[120:], want[120:]).median()) > 2e-4, f"the test would not see {d}"
    r = _runner(folders[case], "float32", chunk_tokens=1)
    (slot,) = r.admit(1)
    assert_rows(r.step([slot], [seq], [list(range(len(seq)))]).cpu(), want, "float32", "in a prompt")
    r.release(slot)
    (slot,) = r.admit(1)
    r.step([slot], [seq[:5]])
    got = [r.step([slot], [[t]]).cpu() for t in seq[5:]]
    assert_rows(torch.cat(got), want[5:], "float32", "decoded alone")
    r.release(slot)


def test_far_keys_and_a_long_decode(tmp_path):
    """Soft scores: a latent layer and an attention layer that see all keys, layers with a window of 500 and of 9.
    Without the keys that lie more than 600 tokens back the oracle's logits move by far more than the tolerance.  In decoding
    a row's keys are cut into shares that are merged (more than 256 keys)."""
    from plain import nuvivik_plain as P
    raw = model(48, 60, [latent(2, 8, 4, 12, 16, 16, 0.1, mlp=None), attention(2, 1, 8, 12, 0.12, 4, softcap=0.7, mlp=None),
                         latent(2, 4, 4, 8, 12, 16, 0.1, window=500, mlp=None),
                         attention(4, 2, 8, 12, 0.3, 8, softcap=2.0, window=9, mlp=None)])
    folder = make_folder(tmp_path, raw, 5, "far")
    cfg, w = oracle_view(folder)
    seq = tokens(70, 700, 60)
    want = P.forward(cfg, w, seq)

    def no_far(i, m):
        return m if m.get("mask") else dict(m, mask={"size": 600})
    assert float(row_errors(P.forward(cfg, w, seq, edit=no_far)[610:], want[610:]).median()) > 1e-4
    for dtype in ("float32", "bfloat16"):
        r = _runner(folder, dtype, chunk_tokens=1)
        (slot,) = r.admit(1)
        got = [r.step([slot], [seq[:580]], [list(range(580))]).cpu()] + [r.step([slot], [[t]]).cpu() for t in seq[580:]]
        assert_rows(torch.cat(got), want, dtype, "far keys")
        r.release(slot)


@pytest.mark.parametrize("name, layer", [
    ("latent", latent(2, 24, 4, 8, 16, 16, 1.0, mlp=None)), ("attention", attention(2, 1, 48, 8, 0.6, 4, mlp=None)),
    ("latent, window", latent(3, 16, 4, 8, 16, 16, 0.6, window=130, mlp=None)),
    ("attention, window", attention(4, 2, 64, 64, 0.3, 16, softcap=12.0, window=130, mlp=None))])
def test_one_key_that_stands_out_inside_and_outside_a_window(tmp_path, name, layer):
    """Models of one layer in which token 1's query is token 0's key (its row is the other's negative, the query's matrix the
    negative of the key's), so that their score carries the softmax.  Token 0 stands once, far back; token 1 asks from page
    borders, from the last place from which a window shows it and from the first from which it does not.  A kernel that lost
    that key (a page, a share, a tile) or kept it one position too long would be off by the size of the logits."""
    from plain import nuvivik_plain as P

    def edit(t):
        t["embed"][1] = -t["embed"][0]
        m = layer["mixer"]
        if layer["type"] == "attention":
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            t["l0.mix.q"] = -t["l0.mix.k"].view(G, d, -1).repeat_interleave(H // G, 0).reshape(H * d, -1)
            t["l0.mix.q.b"] = t["l0.mix.k.b"].view(G, d).repeat_interleave(H // G, 0).reshape(-1)
        else:
            H, d, P_ = m["heads"], m["dim"], m["rot_dim"]
            t["l0.mix.dq"], t["l0.mix.dq.norm"] = -t["l0.mix.dkv"][:m["kv_rank"]], t["l0.mix.dkv.norm"].clone()
            uq = t["l0.mix.uq"].view(H, d + P_, -1)
            uq[:, :d] = t["l0.mix.uk"].view(H, d, -1)
    folder = make_folder(tmp_path, model(32, 40, [layer]), 6, "peak", edit=edit)
    cfg, w = oracle_view(folder)
    far, window = 20, layer["mixer"].get("mask", {}).get("size")
    inside = [far + 40, 63, 64, 128, far + 129] + ([] if window else [290, 299])
    outside = [far + 130, far + 131, 290] if window else []
    seq = [2 + t for t in tokens(71, 300, 38)]
    seq[far] = 0
    for at in inside + outside:
        seq[at] = 1
    want = P.forward(cfg, w, seq)
    other = P.forward(cfg, w, seq[:far] + [2] + seq[far + 1:])
    assert float(row_errors(want[inside], other[inside]).min()) > 5e-2, "the far key does not matter enough"
    if window:
        assert float(row_errors(want[outside], other[outside]).max()) < 1e-12
    for dtype in ("float32", "bfloat16"):
        r = _runner(folder, dtype, chunk_tokens=1)
        (slot,) = r.admit(1)
        whole = r.step([slot], [seq], [list(range(300))]).cpu()
        r.release(slot)
        (slot,) = r.admit(1)
        alone = torch.cat([r.step([slot], [seq[:50]], [list(range(50))]).cpu()] + [r.step([slot], [[t]]).cpu() for t in seq[50:]])
        r.release(slot)
        for got, how in ((whole, "in a prompt"), (alone, "decoded")):
            assert_rows(got, want, dtype, f"{name} {how}")
            assert float(row_errors(got[inside + outside], want[inside + outside]).max()) < (2e-5 if dtype == "float32" else 4e-2), how


def test_every_layer_alone(folders):
    """The residual stream after every layer, in 32-bit, for a prompt; then the same for the prompt's second half fed
    after its first (every mixer resumes from its cache)."""
    from plain import nuvivik_plain as P
    for case in SMALL:
        cfg, w = oracle_view(folders[case])
        seq = tokens(80, 90, cfg["vocab"])
        want = []
        P.forward(cfg, w, seq, taps=want)
        r = _runner(folders[case], "float32")
        (slot,) = r.admit(1)
        taps = r.hidden_states([slot], [seq])[1:]           # the first tap is the embedding
        assert len(taps) == len(want)
        for i, (g, x) in enumerate(zip(taps, want)):
            assert float(row_errors(g.cpu(), x).max()) < 1e-5, f"case {case}: after layer {i}"
        r.release(slot)
        (slot,) = r.admit(1)
        r.step([slot], [seq[:47]])
        taps = r.hidden_states([slot], [seq[47:]])[1:]
        for i, (g, x) in enumerate(zip(taps, want)):
            assert float(row_errors(g.cpu(), x[47:]).max()) < 1e-5, f"case {case}: after layer {i}, second half"
        r.release(slot)


SINGLE = {
    "latent: one head, latents of three and one": latent(1, 4, 2, 5, 1, 3, 0.6, mlp=None),
    "latent: nine heads (two head groups), values wider than keys": latent(9, 8, 4, 24, 24, 40, 0.4, window=50, mlp=None),
    "latent: latents wider than a block's threads": latent(2, 8, 8, 8, 264, 272, 0.2, window=7, mlp=None),
    "latent: a rotated part wider than the rest": latent(3, 2, 40, 6, 16, 12, 0.2, window=100, base=50.0, mlp=None),
    "latent: a window of two": latent(2, 8, 4, 8, 16, 16, 0.5, window=2, mlp=None),
    "attention: keys wider than values, all keys in sight": attention(3, 3, 40, 8, 0.3, 40, mlp=None),
    "attention: heads of 200 and 264 numbers, odd halves": attention(2, 1, 200, 264, 0.05, 66, softcap=3.0, window=50, mlp=None),
    "attention: ten query heads to a kv head": attention(10, 1, 8, 8, 0.7, 2, softcap=4.0, window=100, mlp=None),
    "attention: one head of two numbers, values of three": attention(1, 1, 2, 3, 0.9, 2, softcap=1.0, window=2, mlp=None),
    "attention: a soft-cap far below the scores": attention(4, 2, 16, 16, 1.5, 8, softcap=0.5, mlp=None),
    "attention: eight heads to a kv head, banded, dims of 12": attention(8, 1, 24, 16, 0.5, 12, softcap=50.0, window=65, base=90.0,
                                                                       bands=(5.0, 1.0, 6.0, 80), mlp=None),
    "a dense feed-forward": attention(1, 1, 8, 8, 0.8, 4, window=4),
    "every expert chosen": latent(2, 8, 4, 8, 8, 8, 0.4, mlp=moe(4, 4, 24)),
    "one expert of one": latent(1, 8, 4, 8, 8, 8, 0.4, mlp=moe(1, 1, 40)),
    "forty experts in eight groups, six of three chosen": latent(2, 8, 4, 8, 8, 16, 0.4, mlp=moe(40, 6, 8, groups=(8, 3))),
    "groups of one expert": latent(2, 8, 4, 8, 8, 16, 0.4, mlp=moe(12, 2, 8, groups=(12, 5))),
    "one group": latent(2, 8, 4, 8, 8, 16, 0.4, mlp=moe(9, 3, 16, groups=(1, 1))),
    "experts wider than the model": latent(2, 8, 4, 8, 8, 16, 0.4, mlp=moe(6, 2, 136, groups=(3, 1))),
}


@pytest.mark.parametrize("name", list(SINGLE))
def test_one_layer_models_of_other_sizes(tmp_path, name):
    """Sizes that the kernels' shapes switch on, each as a model of one layer: a prompt, then pieces of one to five
    tokens, in 32-bit; the same in bfloat16."""
    folder = make_folder(tmp_path, model(40, 50, [SINGLE[name]], ff=16, logit_scale=0.5, logit_softcap=3.0), 31, "one")
    seq = tokens(33, 150, 50)
    want = _oracle(folder, [seq])[0]
    for dtype in ("float32", "bfloat16"):
        r = _runner(folder, dtype, chunk_tokens=5)
        (slot,) = r.admit(1)
        got, at = [r.step([slot], [seq[:101]], [list(range(101))]).cpu()], 101
        for k in [1, 1, 2, 5, 1, 3, 1, 1, 4, 30]:
            got.append(r.step([slot], [seq[at:at + k]], [list(range(k))]).cpu())
            at += k
        assert at == len(seq)
        assert_rows(torch.cat(got), want, dtype, name)
        r.release(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wider_layers_and_a_longer_prompt(folders, dtype):
    """A prompt of 500 tokens (windows of 300 and 290: decoding rows see more than 256 keys and are cut into shares), a
    piece of 90, then single tokens beside a second request that starts later.  At these widths and lengths the 32-bit
    rounding noise is larger: every row within 1e-4 of the logits' size and the median within 2e-5."""
    vocab = CASES["E"][0]["vocab"]
    seqs = [tokens(140, 620, vocab), tokens(141, 75, vocab)]
    want = _oracle(folders["E"], seqs)
    r = _runner(folders["E"], dtype, max_seq_len=2048, chunk_tokens=100)
    a, b = r.admit(2)
    probe = list(range(0, 500, 7))
    got = [r.step([a], [seqs[0][:500]], [probe]).cpu(), r.step([a], [seqs[0][500:590]], [list(range(90))]).cpu()]
    out = r.step([b, a], [seqs[1][:60], seqs[0][590:591]], [[59], [0]]).cpu()
    got.append(out[1:2])
    got_b = [out[0:1]]
    for k in range(15):
        out = r.step([a, b], [[seqs[0][591 + k]], [seqs[1][60 + k]]]).cpu()
        got.append(out[0:1])
        got_b.append(out[1:2])
    for k in range(15, 29):
        got.append(r.step([a], [[seqs[0][591 + k]]]).cpu())
    pairs = ((torch.cat(got), torch.cat([want[0][probe], want[0][500:620]])), (torch.cat(got_b), want[1][59:75]))
    for g, x in pairs:
        e = row_errors(g, x)
        if dtype == "float32":
            assert float(e.median()) <= 2e-5 and float(e.max()) <= 1e-4, f"median {float(e.median()):.2e}, worst {float(e.max()):.2e}"
        else:
            assert_rows(g, x, dtype, "wider layers")
    r.release(a)
    r.release(b)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_at_the_tensor_core_kernels_sizes(folders, dtype):
    """Requests of one and two tokens at head sizes that the tensor-core kernels take: a single token at position 0,
    two short prompts side by side, then both decoded, then a prompt of nine tokens beside them."""
    vocab = CASES["E"][0]["vocab"]
    seqs = [tokens(150, 12, vocab), tokens(151, 14, vocab), tokens(152, 9, vocab)]
    want = _oracle(folders["E"], seqs)
    r = _runner(folders["E"], dtype)
    (a,) = r.admit(1)
    got_a = [r.step([a], [seqs[0][:1]]).cpu()]
    (b,) = r.admit(1)
    out = r.step([b, a], [seqs[1][:2], seqs[0][1:3]], [[0, 1], [0, 1]]).cpu()
    got_b, got_a = [out[:2]], got_a + [out[2:]]
    for k in range(9):
        out = r.step([a, b], [[seqs[0][3 + k]], [seqs[1][2 + k]]]).cpu()
        got_a.append(out[0:1])
        got_b.append(out[1:2])
    (c,) = r.admit(1)
    out = r.step([c, b], [seqs[2], seqs[1][11:14]], [list(range(9)), [0, 1, 2]]).cpu()
    got_b.append(out[9:])
    g, x = torch.cat(got_a + got_b + [out[:9]]), torch.cat(want)
    if dtype == "float32":
        e = row_errors(g, x)
        assert float(e.max()) <= 1e-4, f"worst {float(e.max()):.2e}"
    else:
        assert_rows(g, x, dtype, "first tokens")
    for s_ in (a, b, c):
        r.release(s_)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(folders, dtype):
    """The public entry point and its scheduler: more prompts than run side by side, unequal lengths."""
    from plain import nuvivik_plain as P
    from hos_b200 import Engine
    cfg, w = oracle_view(folders["A"])
    prompts = [tokens(100 + i, n, cfg["vocab"]) for i, n in enumerate((5, 70, 1))]
    eng = Engine(folders["A"], dtype=dtype, max_batch=2, max_seq_len=256)
    got = eng.generate_ids(prompts, 10, stop_ids=[])
    for p, g in zip(prompts, got):
        assert len(g) == 10
        seq = list(p)
        for t in g if dtype == "float32" else g[:4]:
            l = P.forward(cfg, w, seq)[-1]
            if dtype == "float32":
                assert float(l.max() - l[t]) < 1e-3, "the chosen token is not the oracle's best"
            else:
                assert float(l.max() - l[t]) < 0.25, "bfloat16 chose a token far from the best"
            seq.append(t)
    eng.runner.cache.check()


def test_the_replay_program_on_a_model_folder(folders, tmp_path):
    vocab = CASES["B"][0]["vocab"]
    seqs = {"x": tokens(110, 80, vocab), "y": tokens(111, 30, vocab), "z": tokens(112, 1, vocab)}
    want = dict(zip(seqs, _oracle(folders["B"], list(seqs.values()))))
    steps, rows = [], {}
    steps.append({"step": 0, "entries": [{"id": "z", "tokens": seqs["z"], "want": [0]}], "end": ["z"]})
    rows[0] = [("z", 0)]
    steps.append({"step": 1, "entries": [{"id": "x", "tokens": seqs["x"][:70], "want": [0, 69]},
                                         {"id": "y", "tokens": seqs["y"][:25], "want": []}], "end": []})
    rows[1] = [("x", 0), ("x", 69)]
    for k in range(10):
        ents = [{"id": "x", "tokens": [seqs["x"][70 + k]], "want": [0]}]
        rws = [("x", 70 + k)]
        if k < 5:
            ents.append({"id": "y", "tokens": [seqs["y"][25 + k]], "want": [0] if k % 2 else []})
            if k % 2:
                rws.append(("y", 25 + k))
        steps.append({"step": 2 + k, "entries": ents, "end": (["y"] if k == 4 else []) + (["x"] if k == 9 else [])})
        rows[2 + k] = rws
    for dtype in ("float32", "bfloat16"):
        out = str(tmp_path / ("out_" + dtype))
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folders["B"], "--dtype", dtype, "--out", out,
                            "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps).encode(),
                           stdout=subprocess.PIPE, stderr=subprocess.PIPE, timeout=900)
        assert p.returncode == 0, p.stderr.decode()[-2000:]
        assert [l for l in p.stdout.decode().splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
        got, ref = [], []
        for n, rws in rows.items():
            got.append(torch.from_numpy(np.fromfile(os.path.join(out, f"{n}.f32"), dtype="<f4").reshape(len(rws), vocab).copy()))
            ref.append(torch.stack([want[i][pos] for i, pos in rws]))
        assert_rows(torch.cat(got), torch.cat(ref), dtype, "replayed steps")


def test_generation_through_the_command_line(folders):
    from plain import nuvivik_plain as P
    cfg, w = oracle_view(folders["C"])
    prompt = tokens(120, 6, cfg["vocab"])
    p = subprocess.run([os.path.join(ROOT, "bin", "hos"), "-m", folders["C"], "--fp32", "--repeat-penalty", "1.0", "-n", "5",
                        "-p", ",".join(map(str, prompt))], stdout=subprocess.PIPE, stderr=subprocess.PIPE, timeout=900)
    assert p.returncode == 0, p.stderr.decode()[-2000:]
    ids = [int(t) for t in p.stdout.decode().strip().split(",")]
    assert ids[:len(prompt)] == prompt and len(ids) == len(prompt) + 5
    seq = list(prompt)
    for t in ids[len(prompt):]:
        l = P.forward(cfg, w, seq)[-1]
        assert float(l.max() - l[t]) < 1e-3
        seq.append(t)


def test_the_attention_kernels_agree_in_bfloat16(folders):
    """The tensor-core kernels against the FMA kernels on the same bfloat16 model: a prompt, a piece, single tokens."""
    from hos_b200.parts.gated_attention import GatedSoftmaxAttention
    from hos_b200.parts.latent_attention import LatentAttention
    vocab = CASES["E"][0]["vocab"]
    seq = tokens(130, 400, vocab)
    outs = []
    for use in (True, False):
        GatedSoftmaxAttention.use_tensor_cores = LatentAttention.use_tensor_cores = use
        try:
            r = _runner(folders["E"], "bfloat16")
            (slot,) = r.admit(1)
            got = [r.step([slot], [seq[:310]], [list(range(0, 310, 3))]), r.step([slot], [seq[310:380]], [list(range(70))])]
            got += [r.step([slot], [[t]]) for t in seq[380:]]
            outs.append(torch.cat(got).cpu())
            r.release(slot)
        finally:
            GatedSoftmaxAttention.use_tensor_cores = LatentAttention.use_tensor_cores = True
    assert_rows(outs[0], outs[1], "bfloat16", "the two kinds of kernel")


def _one_sequence(n, pos0, dev):
    from hos_b200.parts.base import StepInfo
    pos = (pos0 + torch.arange(n)).to(torch.int32).to(dev)
    z = torch.zeros(n, dtype=torch.int32, device=dev)
    return StepInfo(n, 1, None, pos, z, torch.tensor([0, n], dtype=torch.int32, device=dev), z[:1],
                    torch.tensor([pos0 + n], dtype=torch.int32, device=dev), pos0 == 0, n == 1, n, pos0 + n)


def test_the_query_and_key_preparation_alone_against_float64():
    """Rotation in both pairings, part of a head, then a norm without a weight; with a weight before the rotation; neither;
    biases; few rows (wide blocks) and many; the cache's rows in 32-bit."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(2)
    for n, H, G, kd, vd, rot, style, norm in ((37, 3, 1, 24, 16, 8, "rotate_half", "unit"), (700, 4, 2, 64, 128, 64, "rotate_half", "unit"),
                                              (9, 8, 2, 128, 64, 40, "interleaved", "unit"), (5, 2, 2, 200, 12, 66, "rotate_half", "weight"),
                                              (40, 1, 1, 2, 3, 2, "rotate_half", "unit"), (33, 2, 1, 300, 8, 300, "rotate_half", "none"),
                                              (20, 2, 1, 40, 8, 0, "rotate_half", "unit")):
        pages = (n + 63) // 64
        cache = ops.PagedKVArgs(torch.zeros(pages, G, 64, kd, device=dev), torch.zeros(pages, G, 64, vd, device=dev),
                                torch.arange(pages, dtype=torch.int32, device=dev).view(1, -1), 0, G, kd, vd)
        step = _one_sequence(n, 0, dev)
        cols = H * kd + G * (kd + vd)
        proj, bias = torch.randn(n, cols + 3, device=dev), torch.randn(cols, device=dev)
        freq = torch.tensor([90.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64).float().to(dev)
        wq, wk = (torch.randn(kd, device=dev), torch.randn(kd, device=dev)) if norm == "weight" else (None, None)
        q = torch.empty(n, H, kd, device=dev)
        ops.qk_prep(proj, bias, wq, wk, 1e-3, freq if rot else None, rot, 1.0, step, q, cache, H, G, kd, vd,
                    style=ops.ROPE_STYLES[style], unit_norm=norm == "unit")
        x = proj.double().cpu()[:, :cols] + bias.double().cpu()
        ang = torch.arange(n).double()[:, None, None] * freq.double().cpu()
        c, s = torch.cos(ang), torch.sin(ang)

        def prepared(t, w):
            t = t.clone()
            if norm == "weight":
                t = t / torch.sqrt((t * t).mean(-1, keepdim=True) + 1e-3) * w.double().cpu()
            if rot:
                ia = torch.arange(rot // 2) * (1 if style == "rotate_half" else 2)
                ib = ia + (rot // 2 if style == "rotate_half" else 1)
                a, b = t[..., ia].clone(), t[..., ib].clone()
                t[..., ia], t[..., ib] = a * c - b * s, b * c + a * s
            return t / torch.sqrt((t * t).mean(-1, keepdim=True) + 1e-3) if norm == "unit" else t       # after the rotation
        want_q = prepared(x[:, :H * kd].reshape(n, H, kd), wq)
        want_k = prepared(x[:, H * kd:(H + G) * kd].reshape(n, G, kd), wk)
        assert float((q.double().cpu() - want_q).abs().max()) < 2e-4, (n, H, kd, style, norm)
        at = torch.arange(n)
        for g in range(G):
            rows = cache.k_pages[at // 64, g, at % 64].double().cpu()
            if kd % 64 == 0:                                  # the cache's permutation of groups of eight
                rows = torch.stack([torch.cat([rows[t].view(-1, 8)[j ^ (t % 8)] for j in range(kd // 8)]) for t in range(n)])
            assert float((rows - want_k[:, g]).abs().max()) < 2e-4, (n, H, kd, style, norm, "keys")


def test_soft_capped_attention_alone_against_float64():
    """The FMA kernel in one share and several, the tensor-core kernels for prompts and for single tokens, with a soft-cap
    below, at and far above the scores' size and without one."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(8)
    H, G, n = 6, 2, 200
    for kd, vd, cap, window in ((24, 40, 2.0, 70), (64, 128, 1.0, 0), (128, 64, 6.0, 33), (64, 64, 1000.0, 130), (128, 128, 0.0, 64),
                                (128, 128, 3.0, 0)):
        q = (torch.randn(n, H, kd, device=dev)).to(torch.bfloat16).float()
        k, v = torch.randn(n, G, kd).to(torch.bfloat16), torch.randn(n, G, vd).to(torch.bfloat16)
        scale = 3.0 / kd ** 0.5
        s = torch.einsum("ihd,jhd->hij", q.double().cpu(), k.double().repeat_interleave(H // G, 1)) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        i, j = torch.arange(n)[:, None], torch.arange(n)[None]
        s = s.masked_fill(~((i >= j) & ((i - j < window) if window else (i >= j))), float("-inf"))
        want = torch.einsum("hij,jhr->ihr", torch.softmax(s, -1), v.double().repeat_interleave(H // G, 1))
        pages = (n + 63) // 64
        order = torch.randperm(pages + 3)[:pages].to(torch.int32)
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
            kp, vp = (torch.zeros(pages + 3, G, 64, d, device=dev, dtype=dtype) for d in (kd, vd))
            for t in range(n):
                for dst, src, d in ((kp, k, kd), (vp, v, vd)):
                    row = src[t].to(dtype).to(dev).view(G, -1, 8)
                    if d % 64 == 0:
                        row = row[:, [c ^ (t % 8) for c in range(d // 8)]]
                    dst[order[t // 64], :, t % 64] = row.reshape(G, d)
            cache = ops.PagedKVArgs(kp, vp, order.view(1, -1).to(dev).contiguous(), 0, G, kd, vd)
            step = _one_sequence(n, 0, dev)
            runs = {f"{c} shares": (lambda o, c=c: ops.gated_attn(q, cache, None, None, 0, step, o, scale, 0, window, c, softcap=cap) or True)
                    for c in (1, 3)}
            if dtype == torch.bfloat16 and kd % 64 == 0:
                runs["prompt"] = lambda o: ops.gated_attn_mma(q, cache, None, None, 0, step, o, scale, 0, window, 5, softcap=cap)
            for name, run in runs.items():
                out = torch.empty(n, H * vd, device=dev, dtype=dtype)
                assert run(out)
                err = float((out.double().cpu().view(n, H, vd) - want).abs().max())
                assert err < tol * max(1.0, float(want.abs().max())), (kd, vd, cap, window, dtype, name, err)
            if dtype == torch.bfloat16 and kd % 64 == 0:
                one = _one_sequence(1, n - 1, dev)
                for shares in (1, 2):
                    out = torch.empty(1, H * vd, device=dev, dtype=dtype)
                    assert ops.gated_attn_mma_decode(q[n - 1:].contiguous(), cache, None, None, 0, one, out, scale, 0, window, shares,
                                                     softcap=cap)
                    err = float((out.double().cpu().view(H, vd) - want[n - 1]).abs().max())
                    assert err < tol * max(1.0, float(want.abs().max())), (kd, vd, cap, window, "single", shares, err)


def test_the_latent_preparation_alone_against_float64():
    """Both latents' norms, the key part's rotation in both pairings, the cache write (also into a ring), each part with and
    without the other."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(4)
    n, eps = 90, 1e-3
    for R, P, rq, dims, style in ((40, 8, 20, 8, "rotate_half"), (264, 16, 300, 10, "interleaved"), (7, 6, 5, 6, "rotate_half")):
        for dtype in (torch.float32, torch.bfloat16):
            proj = torch.randn(n, rq + R + P + 3, device=dev).to(dtype)
            wc, wq = torch.randn(R, device=dev), torch.randn(rq, device=dev)
            freq = torch.tensor([60.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64).float().to(dev)
            x = proj.double().cpu()
            want_q = x[:, :rq] / torch.sqrt((x[:, :rq] ** 2).mean(-1, keepdim=True) + eps) * wq.double().cpu()
            c = x[:, rq:rq + R]
            kr = x[:, rq + R:rq + R + P].clone()
            ang = torch.arange(n).double()[:, None] * freq.double().cpu()
            ia = torch.arange(dims // 2) * (1 if style == "rotate_half" else 2)
            ib = ia + (dims // 2 if style == "rotate_half" else 1)
            a, b = kr[:, ia].clone(), kr[:, ib].clone()
            kr[:, ia], kr[:, ib] = a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang)
            want_k = torch.cat([c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * wc.double().cpu(), kr], -1)
            tol = (1e-5 if dtype == torch.float32 else 8e-3) * float(want_k.abs().max())
            step = _one_sequence(n, 0, dev)
            for with_q, with_k, ring in ((True, True, 0), (True, False, 0), (False, True, 1)):
                kc, cq = torch.zeros(n, R + P, device=dev, dtype=dtype), torch.zeros(n, rq, device=dev, dtype=dtype)
                pages = torch.zeros(4, 1, 64, R + P, device=dev, dtype=dtype)
                table = torch.tensor([[3, 1]], dtype=torch.int32, device=dev)
                cache = ops.PagedKVArgs(pages, None, table, ring, 1, R + P, 0)
                parts = {}
                if with_q:
                    parts.update(cq=(proj, 0), cq_norm=wq, cq_out=cq)
                if with_k:
                    parts.update(down=(proj, rq), w_norm=wc, kc=kc, cache=cache)
                ops.latent_prep(step, R, P, eps, freq, dims, ops.ROPE_STYLES[style], **parts)
                if with_q:
                    assert float((cq.double().cpu() - want_q).abs().max()) < tol
                if with_k:
                    assert float((kc.double().cpu() - want_k).abs().max()) < tol
                    flat = pages[:, 0]
                    if ring:                      # a ring of one page: it holds the last 64 positions
                        held = torch.stack([flat[3, t % 64] for t in range(26, 90)])
                        assert torch.equal(held, kc[26:]) and float(flat[1].abs().max()) == 0.0
                    else:
                        assert torch.equal(torch.cat([flat[3], flat[1, :26]]), kc)


def test_the_router_with_groups_alone_against_float64():
    """The best groups by their two largest scores, then the largest scores among them; few rows and many, few outputs and
    many, groups of one, logits whose scores round to 1; a row alone and in a batch gives the same numbers."""
    from hos_b200 import ops
    from plain import nuvivik_plain as P
    dev = "cuda"
    torch.manual_seed(19)
    for n, d, n_out, top, count, keep, shift in ((1, 100, 6, 2, 3, 2, 0.0), (17, 1024, 40, 6, 8, 3, 0.0), (70, 250, 12, 3, 4, 2, 0.0),
                                                 (1100, 128, 16, 3, 4, 3, 0.0), (2100, 96, 32, 4, 8, 4, 0.0), (16, 512, 300, 5, 100, 7, 0.0),
                                                 (30, 128, 24, 5, 6, 2, 25.0), (30, 128, 24, 2, 24, 3, 25.0), (30, 128, 24, 5, 6, 2, -25.0)):
        router = torch.randn(n_out, d, device=dev) * (3.0 / d ** 0.5)
        h = torch.randn(n, d, device=dev)
        if shift:                                             # the first column of all: `shift` added to every logit
            router[:, 0] = 1.0
            h[:, 0] = shift
        for dtype in (torch.float32, torch.bfloat16):
            hh = h.to(dtype)
            seq = torch.zeros(n, dtype=torch.int32, device=dev)
            choice = torch.full((n * top,), -7, dtype=torch.int32, device=dev)
            weight = torch.full((n * top,), -7.0, device=dev)
            ops.moe_route(hh, router, None, seq, choice, weight, top, ops.MOE_SCORING["logistic"], groups=(count, keep))
            z = hh.double().cpu() @ router.double().cpu().T
            got, wt = choice.cpu().view(n, top), weight.cpu().view(n, top)
            size, checked = n_out // count, 0
            for r in range(n):
                # a group's standing, a number that grows with the sum of its two largest scores and keeps its digits where
                # the sum is near 2: the sum up to 1, above it one over what is missing to 2 (a group of one: its logit)
                two = z[r].view(count, size).sort(-1, descending=True).values[:, :2]
                total, missing = torch.sigmoid(two).sum(-1), torch.sigmoid(-two).sum(-1)
                stand = two[:, 0] if size == 1 else torch.where(total > 1, 1.0 / missing, total)
                order = sorted(range(count), key=lambda g: (-float(stand[g]), g))
                if keep < count and float(stand[order[keep - 1]] - stand[order[keep]]) < 1e-3 * abs(float(stand[order[keep]])):
                    continue                                  # a close call in 32-bit too
                open_ = [e for e in range(n_out) if e // size in order[:keep]]
                best = sorted(open_, key=lambda e: (-float(z[r, e]), e))
                if len(best) > top and float(z[r, best[top - 1]] - z[r, best[top]]) < 1e-3:
                    continue
                assert sorted(got[r].tolist()) == sorted(best[:top]), (n, n_out, count, r)
                assert float((wt[r].double() - torch.sigmoid(z[r, got[r].long()])).abs().max()) < 1e-5
                checked += 1
                if not shift and dtype == torch.float32 and n < 100:
                    assert sorted(P.choose({"top": top, "groups": {"count": count, "keep": keep}}, torch.sigmoid(z[r]))) == sorted(best[:top])
            assert checked >= 0.8 * n
            c1, w1 = torch.empty(top, dtype=torch.int32, device=dev), torch.empty(top, device=dev)
            ops.moe_route(hh[n - 1:].clone(), router, None, seq[:1], c1, w1, top, ops.MOE_SCORING["logistic"], groups=(count, keep))
            assert torch.equal(c1.cpu(), got[n - 1]) and torch.equal(w1.cpu(), wt[n - 1]), "alone and in a batch differ"
    # other scores: softmax with a correction that steers groups and experts alike
    n, d, n_out, top, count, keep = 20, 64, 12, 2, 4, 2
    router, corr = torch.randn(n_out, d, device=dev) * 0.3, torch.randn(n_out, device=dev) * 0.2
    h = torch.randn(n, d, device=dev)
    choice, weight = torch.empty(n * top, dtype=torch.int32, device=dev), torch.empty(n * top, device=dev)
    ops.moe_route(h, router, corr, torch.zeros(n, dtype=torch.int32, device=dev), choice, weight, top, ops.MOE_SCORING["softmax"],
                  groups=(count, keep))
    s = torch.softmax(h.double().cpu() @ router.double().cpu().T, -1)
    for r in range(n):
        want = P.choose({"top": top, "groups": {"count": count, "keep": keep}}, s[r] + corr.double().cpu())
        got = choice.cpu().view(n, top)[r].tolist()
        assert got == want and float((weight.cpu().view(n, top)[r].double() - s[r, got]).abs().max()) < 1e-5


def test_the_square_of_relu_experts_alone_against_float64():
    """The ungated experts' up product: tiles on the tensor cores, plain tiles, 32-bit, and the kernels for a handful of
    pairs with one, two or four features to a warp; the weight on the output and on the input."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(23)
    act = ops.EXPERT_ACTIVATIONS["relu_square"]
    tile = ops.moe_tile_rows()
    for rows, top, E, d, f, dtype, few, on_input in ((1, 3, 9, 1024, 1024, torch.bfloat16, True, False), (4, 2, 5, 1000, 2040, torch.bfloat16, True, False),
                                                     (8, 4, 6, 520, 4104, torch.bfloat16, True, True), (150, 2, 5, 264, 136, torch.bfloat16, False, False),
                                                     (70, 3, 4, 100, 36, torch.bfloat16, False, True), (40, 2, 7, 72, 50, torch.float32, False, False)):
        pairs = rows * top
        h = torch.randn(rows, d, device=dev).to(dtype)
        up = (torch.randn(E, f, d, device=dev) / d ** 0.5).to(dtype)
        down = (torch.randn(E, d, f, device=dev) / f ** 0.5).to(dtype)
        choice = torch.stack([torch.randperm(E)[:top] for _ in range(rows)]).to(torch.int32).view(-1).to(dev)
        weight = torch.rand(pairs, device=dev) + 0.25
        out = torch.zeros(pairs, d, device=dev)
        if few:
            y = torch.zeros(pairs, f, dtype=dtype, device=dev)
            assert ops.moe_few(h, up, down, choice, weight, y, out, top, E, 0.0, 1.0, 0.0, on_input, act)
        else:
            tiles = min(pairs, E) + pairs // tile
            listed, owner = (torch.empty(k, dtype=torch.int32, device=dev) for k in (tiles * tile, tiles))
            ops.moe_align(choice, E, listed, owner)
            y = torch.empty(tiles * tile, f, dtype=dtype, device=dev)
            ops.moe_gate_up(h, up, listed, owner, y, top, 0.0, 1.0, 0.0, weight if on_input else None, act)
            ops.moe_down(y, down, listed, owner, None if on_input else weight, out)
        tol = 1e-5 if dtype == torch.float32 else 2e-2
        for p in range(pairs):
            e, x, wt = int(choice[p]), h[p // top].double().cpu(), float(weight[p])
            z = torch.relu(up[e].double().cpu() @ (x * wt if on_input else x)) ** 2
            want = down[e].double().cpu() @ z * (1.0 if on_input else wt)
            assert float((out[p].double().cpu() - want).abs().max()) < tol * max(1e-2, float(want.abs().max())), (rows, d, f, p)


def test_products_with_an_activation_and_no_bias():
    """act(x . W^T) with the tanh-form GELU and no bias in every product: few rows, the tcgen05 kernel in both orientations
    and on pairs of SMs, the plain kernel in both types; with a bias as well."""
    from hos_b200 import ops
    from hos_b200.parts import linear
    from plain import nuvivik_plain as P
    dev = "cuda"
    torch.manual_seed(13)
    act = ops.BIAS_ACTIVATIONS["gelu_tanh"]
    for m, n, k, dtype in ((3, 80, 256, torch.bfloat16), (30, 264, 136, torch.bfloat16), (100, 320, 256, torch.bfloat16),
                           (700, 520, 320, torch.bfloat16), (65, 40, 50, torch.bfloat16), (20, 70, 33, torch.float32)):
        x = torch.randn(m, k, device=dev).to(dtype)
        w = (torch.randn(n, k, device=dev) * 2.0 / k ** 0.5).to(dtype)
        b = torch.randn(n, device=dev)
        for bias in (None, b):
            z = x.double().cpu() @ w.double().cpu().T + (b.double().cpu() if bias is not None else 0.0)
            want = P.gelu_tanh(z)
            got = linear.matmul(x, w, epilogue=ops.EPI_BIAS, act=act, bias=bias).double().cpu()
            tol = 1e-5 if dtype == torch.float32 else 2e-2
            assert float((got - want).abs().max()) < tol * float(want.abs().max()), (m, n, k, dtype, bias is not None)
        # large negative inputs vanish, large positive ones pass
        one = linear.matmul(x * 0 + 50.0, torch.cat([w * 0 + 1.0, w * 0 - 1.0]), epilogue=ops.EPI_BIAS, act=act)
        assert bool((one[:, :n] > 40.0).all()) and float(one[:, n:].abs().max()) == 0.0


def test_a_norm_added_to_the_stream_with_the_stream_itself_on_the_way_out():
    """x += norm(y) and x in the products' type from the same launch, for few rows, many rows and widths of every path; y in
    rows of both types and as partial sums."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(3)
    for n, d, parts, ydt in ((3, 72, 1, torch.bfloat16), (300, 256, 1, torch.bfloat16), (5, 101, 1, torch.float32), (2, 4096, 4, torch.float32),
                             (400, 512, 3, torch.float32), (7, 6000, 1, torch.bfloat16)):
        y = torch.randn(*((parts, n, d) if parts > 1 else (n, d)), device=dev).to(ydt)
        x, w = torch.randn(n, d, device=dev), torch.randn(d, device=dev)
        y64 = y.double().cpu().sum(0) if parts > 1 else y.double().cpu()
        want = x.double().cpu() + y64 / torch.sqrt((y64 * y64).mean(-1, keepdim=True) + 1e-4) * w.double().cpu()
        h = torch.empty(n, d, dtype=torch.bfloat16, device=dev)
        ops.norm_add_norm(y, w, 1e-4, False, x, h=h)
        assert float((x.double().cpu() - want).abs().max()) < 1e-5 * float(want.abs().max())
        assert torch.equal(h, x.to(torch.bfloat16))
