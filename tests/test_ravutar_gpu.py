"""Ravutar on the GPU against the plain oracle (tests/plain/ravutar_plain.py): every mechanism alone, whole prompts,
decoding through the cache and the states, prompts in pieces, batches against each request alone, reuse of slots, pages
and states, the steps of the query factor, the first tokens, far keys and long memories, other sizes, and generation
through the engine, the replay program and the command line."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from ravutar_cases import CASES, assert_rows, left, make_folder, mamba2, model, oracle_view, parallel, right, row_errors, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("ravutar")
    return {k: make_folder(base, raw, seed, k) for k, (raw, seed) in CASES.items()}


def _runner(folder, dtype, **kw):
    from hos_b200.engine import Runner
    kw.setdefault("max_tokens", 4096)
    kw.setdefault("max_seq_len", 1024)
    return Runner.from_folder(folder, dtype=dtype, **kw)


def _oracle(folder, seqs):
    from plain import ravutar_plain as P
    cfg, w = oracle_view(folder)
    return [P.forward(cfg, w, s) for s in seqs]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["A", "B", "C", "D"])
def test_whole_prompts_of_unequal_lengths(folders, case, dtype):
    vocab = CASES[case][0]["vocab"]
    seqs = [tokens(i, n, vocab) for i, n in enumerate((1, 2, 37, 150))]      # 1, 2: fewer than the taps; 150: beyond two pages
    want = _oracle(folders[case], seqs)
    r = _runner(folders[case], dtype)
    slots = r.admit(len(seqs))
    got = r.step(slots, seqs, [list(range(len(s))) for s in seqs]).cpu()
    assert_rows(got, torch.cat(want), dtype, f"case {case}")
    for s in slots:
        r.release(s)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["A", "B", "C", "D"])
def test_a_prompt_then_token_by_token(folders, case, dtype):
    """Two requests decoded side by side through the replayed single-token step, across page borders (64, 128) and every
    step of the query factor; the shorter one leaves first.  The longer one is decoded for 141 steps, so convolution
    inputs and matrix states are carried for as long."""
    vocab = CASES[case][0]["vocab"]
    seqs = [tokens(20, 150, vocab), tokens(21, 90, vocab)]
    plens = [9, 61]
    want = _oracle(folders[case], seqs)
    r = _runner(folders[case], dtype)
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


@pytest.mark.parametrize("case, dtype", [("A", "float32"), ("A", "bfloat16"), ("B", "float32"), ("C", "float32"), ("D", "float32"),
                                         ("D", "bfloat16")])
def test_a_prompt_in_pieces_of_many_sizes(folders, case, dtype):
    """Pieces down to two tokens and one (fewer than the taps: kept inputs come from two pieces back), pieces that end on a
    page's border and one past it: convolutions and matrix states go on from what the slot holds."""
    vocab = CASES[case][0]["vocab"]
    seq = tokens(30, 230, vocab)
    want = _oracle(folders[case], [seq])[0]
    r = _runner(folders[case], dtype)
    (slot,) = r.admit(1)
    at, got = 0, []
    for k in [2, 3, 59, 1, 65, 7, 2, 40, 1, 1, 30, 2, 2, 15]:
        piece = seq[at:at + k]
        got.append(r.step([slot], [piece], [list(range(len(piece)))]).cpu())
        at += len(piece)
    assert at == len(seq)
    assert_rows(torch.cat(got), want, dtype, f"case {case}")
    r.release(slot)
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["A", "D"])
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


def test_slots_pages_and_states_that_are_freed_are_used_again(folders):
    """What a freed slot's pages, convolution inputs and matrix states still hold must never be read."""
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
            t.fill_(1e4)
    for t in r.cache.state_tensors():
        t.fill_(77)
    (again,) = r.admit(1)
    assert again == slot
    got = [r.step([again], [second[:70]], [list(range(70))]).cpu()]
    for t in second[70:]:
        got.append(r.step([again], [[t]]).cpu())
    assert_rows(torch.cat(got), want, "float32", "second request in a used slot")
    r.release(again)
    # a request that starts with single tokens in a used slot: its states start at zero all the same
    for t in r.cache.state_tensors():
        t.fill_(77)
    (again,) = r.admit(1)
    got = [r.step([again], [[t]]).cpu() for t in second[:12]]
    assert_rows(torch.cat(got), want[:12], "float32", "token by token from the first in a used slot")
    r.release(again)
    # two slots whose requests swap: each goes on from its own states
    a, b = r.admit(2)
    r.step([a, b], [second[:20], first[:9]])
    got = [r.step([b, a] if k % 2 else [a, b], [[first[9 + k]], [second[20 + k]]] if k % 2 else [[second[20 + k]], [first[9 + k]]]).cpu()
           for k in range(6)]
    assert_rows(torch.cat([g[1 if k % 2 else 0:][:1] for k, g in enumerate(got)]), want[20:26], "float32", "rows that change places")
    r.release(a)
    r.release(b)
    r.cache.check()


@pytest.mark.parametrize("case", ["A", "C", "D"])
def test_the_steps_of_the_query_factor_in_prompts_and_in_decoding(folders, case):
    """The oracle whose factor steps one position earlier or later is far from the oracle itself at the very positions
    where they differ, and the library agrees with the oracle at every position, in a prompt and alone."""
    from plain import ravutar_plain as P
    cfg, w = oracle_view(folders[case])
    seq = tokens(60, 140, cfg["vocab"])
    want = P.forward(cfg, w, seq)
    for i, layer in enumerate(cfg["layers"]):
        t = layer["mixer"].get("left", {}).get("q_temp")
        if not t or t["every"] < 3:
            continue
        # the same factor, taken at p instead of at p + 1: only the positions just before a step differ
        P_factor = P.query_factor
        P.query_factor = lambda q, p: P_factor(q, p - 1) if q == t else P_factor(q, p)
        try:
            late = P.forward(cfg, w, seq)
        finally:
            P.query_factor = P_factor
        edge = t["every"] - 1                    # the first position with the second value
        assert float(row_errors(late, want)[:edge].max()) < 1e-12, "positions before the first step do not differ"
        assert float(row_errors(late, want)[edge]) > 2e-4, "the test would not see the step"
    r = _runner(folders[case], "float32")
    (slot,) = r.admit(1)
    assert_rows(r.step([slot], [seq], [list(range(len(seq)))]).cpu(), want, "float32", "in a prompt")
    r.release(slot)
    (slot,) = r.admit(1)
    got = [r.step([slot], [[t]]).cpu() for t in seq]
    assert_rows(torch.cat(got), want, "float32", "decoded alone, from the first token")
    r.release(slot)


def test_far_keys_the_sink_and_long_memories(tmp_path):
    """Soft scores and slow decays on both kinds of state: without the keys that lie more than 600 tokens back, without the
    one in the denominator, or with a state that forgets faster, the oracle's logits move by far more than the
    tolerance.  In decoding a row's keys are cut into shares that are merged (more than 256 keys)."""
    from plain import ravutar_plain as P
    raw = model(48, 60, [parallel(left(2, 1, 8, 12, 0.15, 3, (0.2, 50)), right(2, 8, 12, 400.0, 4), mlp=None),
                         mamba2(2, 12, 8, 1, 4, 1, mlp=None),
                         parallel(left(4, 2, 8, 12, 0.1, 2), right(1, 12, 8, 900.0, 3), mlp=None)], streams=2)

    def edit(t):
        t["l1.mix.A_log"].fill_(-6.0)                    # exp(-exp(-6) softplus(..)): about two thousandths per token
        for i in (0, 2):
            t[f"l{i}.mix.left.v"] *= 3.0
            t[f"l{i}.mix.left.q"] *= 0.4
    folder = make_folder(tmp_path, raw, 5, "far", edit=edit)
    cfg, w = oracle_view(folder)
    seq = tokens(70, 644, 60)
    want = P.forward(cfg, w, seq)

    def no_far(i, m):
        return dict(m, left=dict(m["left"], only_last=600)) if "left" in m else m

    def no_sink(i, m):
        return dict(m, left=dict(m["left"], no_sink=True)) if "left" in m else m

    def forgets(i, m):
        return dict(m, right=dict(m["right"], tau=m["right"]["tau"] / 8)) if "right" in m else m
    assert float(row_errors(P.forward(cfg, w, seq, edit=no_far)[610:], want[610:]).median()) > 1e-4
    assert float(row_errors(P.forward(cfg, w, seq, edit=no_sink)[610:], want[610:]).median()) > 1e-4
    assert float(row_errors(P.forward(cfg, w, seq, edit=forgets)[610:], want[610:]).median()) > 2e-3
    faster = dict(w, **{"l1.mix.A_log": w["l1.mix.A_log"] + 1.0})
    assert float(row_errors(P.forward(cfg, faster, seq)[610:], want[610:]).median()) > 2e-3
    for dtype in ("float32", "bfloat16"):
        r = _runner(folder, dtype)
        (slot,) = r.admit(1)
        got = [r.step([slot], [seq[:600]], [list(range(600))]).cpu()] + [r.step([slot], [[t]]).cpu() for t in seq[600:]]
        assert_rows(torch.cat(got), want, dtype, "far keys and long memories")
        r.release(slot)


def test_one_key_far_back_that_stands_out(tmp_path):
    """A key among hundreds made to carry the softmax: the rows of its token and of the asking tokens are scaled so that
    their score stands out; a kernel that lost that key (a page, a share, a tile) would be off by the size of the logits."""
    from plain import ravutar_plain as P
    raw = model(32, 40, [parallel(left(2, 1, 8, 8, 0.5, 1, (0.5, 64)), right(1, 8, 8, 2.0, 4), (2.0, 0.3), mlp=None)], streams=2)
    seq = tokens(71, 400, 40)
    seq = [t if t not in (7, 11) else 5 for t in seq]
    seq[3] = 7
    for t in range(380, 400):
        seq[t] = 11

    def edit(t):
        # every query of token 11 is a multiple of token 7's key: the score of the pair is large, all others are small
        for r in ("q", "k"):
            t[f"l0.mix.left.{r}.conv"].fill_(1.0)
            t[f"l0.mix.left.{r}.b"].zero_()
        e7, e11, s = t["embed"][7], t["embed"][11], t["l0.hc1.in"].sum()
        h7, h11 = s * e7 * t["l0.norm1"], s * e11 * t["l0.norm1"]
        h7, h11 = h7 / h7.norm() * 32 ** 0.5, h11 / h11.norm() * 32 ** 0.5
        k = t["l0.mix.left.k"] @ h7
        k = k / k.norm()
        t["l0.mix.left.k"] += torch.outer(k * 4.0, h7) / 32
        for h in range(2):
            t["l0.mix.left.q"][h * 8:(h + 1) * 8] += torch.outer(k * 5.0, h11) / 32
    folder = make_folder(tmp_path, raw, 6, "peak", edit=edit)
    cfg, w = oracle_view(folder)
    want = P.forward(cfg, w, seq)
    cut = P.forward(cfg, w, seq[:3] + [8] + seq[4:])
    assert float(row_errors(cut[380:], want[380:]).median()) > 1e-2, "the far key does not matter enough"
    for dtype in ("float32", "bfloat16"):
        r = _runner(folder, dtype)
        (slot,) = r.admit(1)
        got = [r.step([slot], [seq[:390]], [list(range(370, 390))]).cpu()] + [r.step([slot], [[t]]).cpu() for t in seq[390:]]
        assert_rows(torch.cat(got), want[370:], dtype, "a far key that stands out")
        r.release(slot)


def test_every_layer_run_alone(folders):
    """The sum of the streams after every layer run (a looped layer counts each time), in 32-bit, for a prompt; then the
    same for the prompt's second half fed after the first (every run resumes from its own cache and states)."""
    from plain import ravutar_plain as P
    for case in ("A", "B", "C", "D"):
        cfg, w = oracle_view(folders[case])
        seq = tokens(80, 90, cfg["vocab"])
        want = []
        P.forward(cfg, w, seq, taps=want)
        r = _runner(folders[case], "float32")
        (slot,) = r.admit(1)
        taps = r.hidden_states([slot], [seq])[1:]           # the first tap is the embedding
        assert len(taps) == len(want) == len(P.run_order(cfg))
        for i, (g, x) in enumerate(zip(taps, want)):
            assert float(row_errors(g.cpu(), x).max()) < 2e-5, f"case {case}: after layer run {i}"
        r.release(slot)
        (slot,) = r.admit(1)
        r.step([slot], [seq[:47]])
        taps = r.hidden_states([slot], [seq[47:]])[1:]
        for i, (g, x) in enumerate(zip(taps, want)):
            assert float(row_errors(g.cpu(), x[47:]).max()) < 2e-5, f"case {case}: after layer run {i}, second half"
        r.release(slot)


R0 = right(1, 8, 8, 4.0, 2)
L0 = left(1, 1, 8, 8, 0.3, 2)
SINGLE = {
    "attention alone (the other side times zero)": (parallel(left(3, 3, 12, 20, 0.5, 3, (0.6, 10)), R0, (1.0, 0.0), mlp=None), 2),
    "linear attention alone": (parallel(L0, right(3, 20, 12, 16.0, 6), (0.0, 1.0), mlp=None), 2),
    "attention: keys of 200 numbers, values of 264": (parallel(left(2, 1, 200, 264, 0.05, 4), R0, mlp=None), 1),
    "attention: ten query heads to a kv head, sixteen taps": (parallel(left(10, 1, 8, 8, 0.5, 16, (1.0, 5)), R0, mlp=None), 3),
    "attention: one head of one number": (parallel(left(1, 1, 1, 3, 0.9, 2, (0.1, 1)), R0, mlp=None), 2),
    "attention without a convolution": (parallel({k: v for k, v in L0.items() if k != "conv"}, R0, mlp=None), 2),
    "linear attention: a key of one number, values of three": (parallel(L0, right(2, 1, 3, 1.0, 1), mlp=None), 2),
    "linear attention: keys of 200, values of 40, rank 33": (parallel(L0, right(2, 200, 40, 16.0, 33), mlp=None), 2),
    "linear attention: keys of 300": (parallel(L0, right(1, 300, 8, 8.0, 4), mlp=None), 2),
    "linear attention: values of 264, tau below one": (parallel(L0, right(3, 8, 264, 0.5, 4), mlp=None), 2),
    "state space: one head of one number, a state of one": (mamba2(1, 1, 1, 1, 1, 1, mlp=None), 2),
    "state space: a state of 200, heads of 36, a norm part that cuts heads": (mamba2(3, 36, 200, 1, 4, 4, mlp=None), 2),
    "state space: a state of 600 and sixteen taps": (mamba2(2, 8, 600, 2, 16, 1, mlp=None), 2),
    "state space: a group to a head, a norm part to a head": (mamba2(5, 12, 10, 5, 2, 5, mlp=None), 2),
    "state space: an inner size of 1,280 in one part": (mamba2(10, 128, 16, 2, 4, 1, mlp=None), 2),
    "seven streams": (mamba2(2, 8, 8, 1, 3, 2), 7),
    "sixteen streams": (parallel(L0, R0), 16),
    "one stream and no feed-forward": (parallel(L0, R0, mlp=None), 1),
    "a feed-forward wider than the model": (mamba2(2, 8, 8, 2, 3, 1, mlp={"kind": "dense", "ff": 264}), 4),
}


@pytest.mark.parametrize("name", list(SINGLE))
def test_one_layer_models_of_other_sizes(tmp_path, name):
    """Sizes that the kernels' shapes switch on, each as a model of one layer (and its mechanisms alone): a prompt, then
    pieces of one to five tokens, in 32-bit."""
    layer, streams = SINGLE[name]
    raw = model(40, 50, [layer], streams, ff=16, eps=1e-4)
    folder = make_folder(tmp_path, raw, 31, "one")
    seq = tokens(33, 150, 50)
    want = _oracle(folder, [seq])[0]
    r = _runner(folder, "float32")
    (slot,) = r.admit(1)
    got, at = [r.step([slot], [seq[:101]], [list(range(101))]).cpu()], 101
    for k in [1, 1, 2, 5, 1, 3, 1, 1, 4, 30]:
        got.append(r.step([slot], [seq[at:at + k]], [list(range(k))]).cpu())
        at += k
    assert at == len(seq)
    assert_rows(torch.cat(got), want, "float32", name)
    r.release(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wider_layers_and_a_longer_prompt(folders, dtype):
    """A prompt of 700 tokens (decoding rows see more than 256 keys and are cut into shares), a piece of 90, then single
    tokens beside a second request that starts later.  At these widths and lengths the 32-bit rounding noise is larger:
    every row within 1e-4 of the logits' size and the median within 2e-5."""
    vocab = CASES["E"][0]["vocab"]
    seqs = [tokens(140, 820, vocab), tokens(141, 75, vocab)]
    want = _oracle(folders["E"], seqs)
    r = _runner(folders["E"], dtype, max_seq_len=2048)
    a, b = r.admit(2)
    probe = list(range(0, 700, 7))
    got = [r.step([a], [seqs[0][:700]], [probe]).cpu(), r.step([a], [seqs[0][700:790]], [list(range(90))]).cpu()]
    out = r.step([b, a], [seqs[1][:60], seqs[0][790:791]], [[59], [0]]).cpu()
    got.append(out[1:2])
    got_b = [out[0:1]]
    for k in range(15):
        out = r.step([a, b], [[seqs[0][791 + k]], [seqs[1][60 + k]]]).cpu()
        got.append(out[0:1])
        got_b.append(out[1:2])
    for k in range(15, 29):
        got.append(r.step([a], [[seqs[0][791 + k]]]).cpu())
    pairs = ((torch.cat(got), torch.cat([want[0][probe], want[0][700:820]])), (torch.cat(got_b), want[1][59:75]))
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
    for g, x in ((torch.cat(got_a), want[0]), (torch.cat(got_b), want[1]), (out[:9], want[2])):
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
    from plain import ravutar_plain as P
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
    from plain import ravutar_plain as P
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
    vocab = CASES["E"][0]["vocab"]
    seq = tokens(130, 400, vocab)
    outs = []
    for use in (True, False):
        GatedSoftmaxAttention.use_tensor_cores = use
        try:
            r = _runner(folders["E"], "bfloat16")
            (slot,) = r.admit(1)
            got = [r.step([slot], [seq[:310]], [list(range(0, 310, 3))]), r.step([slot], [seq[310:380]], [list(range(70))])]
            got += [r.step([slot], [[t]]) for t in seq[380:]]
            outs.append(torch.cat(got).cpu())
            r.release(slot)
        finally:
            GatedSoftmaxAttention.use_tensor_cores = True
    assert_rows(outs[0], outs[1], "bfloat16", "the two kinds of kernel")


# ---- kernels alone ---------------------------------------------------------------------------------------------------

def _ragged(dev, lens, starts, slots):
    """A StepInfo of sequences of these lengths that go on from these positions, with a padding row at the end."""
    from hos_b200.parts.base import StepInfo
    n = sum(lens)
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    pos = i32([s + t for k, s in zip(lens, starts) for t in range(k)] + [0])
    seq = i32([i for i, k in enumerate(lens) for _ in range(k)] + [-1])
    return StepInfo(n + 1, len(lens), None, pos, seq, i32(cu), i32(slots), i32([s + k for k, s in zip(lens, starts)]), False, False,
                    max(lens), max(s + k for k, s in zip(lens, starts))), cu


@pytest.mark.parametrize("taps, c, act", [(4, 64, "x_logistic"), (3, 30, "none"), (2, 260, "x_logistic"), (1, 8, "x_logistic"),
                                          (7, 12, "none"), (16, 5, "x_logistic")])
def test_the_convolution_kernel_alone(taps, c, act):
    """Sequences that start and that go on, shorter and longer than the taps and than a thread's run of rows, in float64;
    the kept inputs afterwards, also when the sequences bring single tokens; the step sizes in the same launch."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(4)
    H, col = 5, 4
    for lens, starts in (([1, 40, 2, 300, 17], [0, 9, 0, 0, 3]), ([1, 1, 1, 1], [0, 7, 1, 200])):
        step, cu = _ragged(dev, lens, starts, [6, 0, 3, 5, 2][:len(lens)])
        n, ld = sum(lens) + 1, -(-(col + c + H) // 4) * 4
        raw = torch.randn(n, ld, device=dev)
        w, b, ib = torch.randn(taps, c, device=dev), torch.randn(c, device=dev), torch.randn(c, device=dev)
        keep = torch.randn(7, taps - 1, c, device=dev)
        dt_bias, a_log = torch.randn(H, device=dev), torch.randn(H, device=dev)
        out, dt, g = torch.empty(n, c, device=dev), torch.empty(n, H, device=dev), torch.empty(n, H, device=dev)
        single = max(lens) == 1
        kept = keep.clone()
        ops.conv_act_rows(raw, col, w, b, kept, act, step, out, single, (col + c, dt_bias, a_log, dt, g), in_bias=ib)
        if not single:
            ops.conv_keep(raw, taps, kept, step, c, col, ib)
        U, W = (raw[:, col:col + c] + ib).double().cpu(), w.double().cpu().T
        for i, k in enumerate(lens):
            slot = int(step.seq_slot[i])
            before = keep[slot].double().cpu() if starts[i] else torch.zeros(taps - 1, c, dtype=torch.float64)
            seq = torch.cat([before, U[cu[i]:cu[i + 1]]])
            y = torch.stack([(seq[t:t + taps].T * W).sum(1) for t in range(k)]) + b.double().cpu()
            if act == "x_logistic":
                y = y * torch.sigmoid(y)
            assert float((out[cu[i]:cu[i + 1]].double().cpu() - y).abs().max()) < 1e-5 * max(1.0, float(y.abs().max()))
            if taps > 1:
                assert torch.equal(kept[slot].double().cpu(), seq[k:k + taps - 1].float().double())
        for slot in set(range(7)) - set(step.seq_slot.tolist()):
            assert torch.equal(kept[slot], keep[slot]), "another slot's inputs were touched"
        want = torch.nn.functional.softplus(raw.double().cpu()[:-1, col + c:col + c + H] + dt_bias.double().cpu(), threshold=1e9)
        assert float((dt[:-1].double().cpu() - want).abs().max()) < 1e-5
        assert float((g[:-1].double().cpu() - torch.exp(-torch.exp(a_log.double().cpu()) * want)).abs().max()) < 1e-5
        assert float(out[-1].abs().max()) == 0.0 and float(dt[-1].abs().max()) == 0.0, "a padding row is zeros"


@pytest.mark.parametrize("H, G, d, vd", [(3, 3, 16, 20), (4, 2, 64, 48), (2, 1, 200, 8), (1, 1, 7, 5)])
def test_the_scan_rules_alone(H, G, d, vd):
    """The decay rule with decays and factors on v per token, grouped keys, and the rule with a decay per key channel (keys
    not grouped there), with a constant on the read-outs, over sequences that start and go on, against float64."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(5)
    lens, starts = [1, 30, 9], [0, 0, 12]
    step, cu = _ragged(dev, lens, starts, [2, 0, 3])
    n = sum(lens) + 1
    for channel in (False, True):
        g_heads = H if channel else G
        ld = -(-(2 * g_heads * d + H * vd + 3) // 4) * 4
        rows = torch.randn(n, ld, device=dev) * 0.5
        g = torch.rand(n, H * d if channel else H, device=dev) * 0.5 + 0.5
        f = None if channel else torch.rand(n, H, device=dev) + 0.3
        state = torch.randn(4, H, vd, d, device=dev)
        kept = state.clone()
        out = torch.empty(n, H * vd, device=dev)
        ops.state_scan(rows, 0, g_heads * d, 2 * g_heads * d, False, g, True, None, kept, step, out, H, g_heads, d, vd, v_factor=f,
                       channel_g=channel, o_mult=0.3)
        X = rows.double().cpu()
        for i, k in enumerate(lens):
            slot = int(step.seq_slot[i])
            for h in range(H):
                kh = h // (H // g_heads)
                S = state[slot, h].double().cpu().T.clone() if starts[i] else torch.zeros(d, vd, dtype=torch.float64)
                for t in range(cu[i], cu[i + 1]):
                    q, key = X[t, kh * d:(kh + 1) * d], X[t, (g_heads + kh) * d:(g_heads + kh + 1) * d]
                    v = X[t, 2 * g_heads * d + h * vd:2 * g_heads * d + (h + 1) * vd]
                    if channel:
                        S = g[t, h * d:(h + 1) * d].double().cpu()[:, None] * S + torch.outer(key, v)
                    else:
                        S = float(g[t, h]) * S + float(f[t, h]) * torch.outer(key, v)
                    want = 0.3 * (S.T @ q)
                    got = out[t, h * vd:(h + 1) * vd].double().cpu()
                    assert float((got - want).abs().max()) < 2e-5 * max(1.0, float(want.abs().max())), (channel, i, h, t)
                assert float((kept[slot, h].double().cpu().T - S).abs().max()) < 2e-5 * max(1.0, float(S.abs().max()))


def test_the_row_kernels_alone():
    """The decay per key channel, the skip with its gate before the norm, the streams' update with the next norm (one to
    sixteen streams, a branch in either type or as partial sums, with and without a bias, widths of no multiple of four),
    the sum of the streams, the norm-and-gate into columns of a wider row, all against float64."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(6)
    n = 37
    seq = torch.zeros(n, dtype=torch.int32, device=dev)
    seq[5] = -1
    for rank, c, tau in ((1, 7, 1.0), (24, 300, 16.0), (130, 64, 0.5)):
        rows = torch.randn(n, rank + 9, device=dev) * 3
        w, b = torch.randn(rank, c, device=dev), torch.randn(c, device=dev) * 4
        out = torch.empty(n, c, device=dev)
        ops.channel_decay(rows, 6, rank, w, b, tau, out)
        z = rows.double().cpu()[:, 6:6 + rank] @ w.double().cpu() + b.double().cpu()
        want = torch.exp(torch.nn.functional.logsigmoid(z) / tau)
        assert float((out.double().cpu() - want).abs().max()) < 2e-5, (rank, c)
    for H, vd, parts, xl, zl in ((3, 36, 4, 5, 3), (8, 64, 4, 4, 8), (10, 128, 1, 0, 0), (1, 3, 1, 1, 2), (40, 128, 1, 0, 4), (64, 128, 2, 0, 0),
                                 (6, 12, 9, 4, 4)):
        inner = H * vd
        o, x, z = (torch.randn(n, inner + e, device=dev) for e in (0, 2 * xl, 2 * zl))
        skip, w = torch.randn(H, device=dev), torch.randn(inner, device=dev)
        y = o.double().cpu() + skip.double().cpu().repeat_interleave(vd) * x.double().cpu()[:, xl:xl + inner]
        zz = z.double().cpu()[:, zl:zl + inner]
        y = (y * zz * torch.sigmoid(zz)).view(n, parts, inner // parts)
        y = (y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-3)).reshape(n, inner) * w.double().cpu()
        y[5] = 0.0
        for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
            out = torch.empty(n, inner, device=dev, dtype=dt)
            ops.skip_gate_norm(o, x, xl, skip, z, zl, w, 1e-3, seq, out, H, vd, parts)
            assert float((out.double().cpu() - y).abs().max()) < tol * max(1.0, float(y.abs().max())), (H, vd, parts)
    for S, D in ((1, 64), (2, 33), (3, 100), (4, 4096), (4, 30), (5, 64), (16, 20)):
        x = torch.randn(n, S * D, device=dev)
        mix, ow, iw = torch.randn(S, S, device=dev), torch.randn(S, device=dev), torch.randn(S, device=dev)
        w, bias = torch.randn(D, device=dev), torch.randn(D, device=dev)
        X = x.double().cpu().view(n, S, D)
        for y, b, use_in in ((torch.randn(n, D, device=dev), bias, True), (torch.randn(n, D, device=dev).to(torch.bfloat16), None, True),
                             (torch.randn(3, n, D, device=dev), bias, False), (None, None, True)):
            x2 = x.clone()
            new = X
            if y is not None:
                Y = y.double().cpu()
                Y = Y.sum(0) if Y.dim() == 3 else Y
                if b is not None:
                    Y = Y + b.double().cpu()
                new = torch.einsum("st,nsd->ntd", mix.double().cpu(), X) + ow.double().cpu()[None, :, None] * Y[:, None]
            u = (new * (iw.double().cpu() if use_in else torch.ones(S, dtype=torch.float64))[None, :, None]).sum(1)
            h = u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-4) * w.double().cpu()
            for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
                x2.copy_(x)
                hh = torch.empty(n, D, device=dev, dtype=dt)
                ops.hyper_norm(x2, S, y=y, bias=b, mix=mix if y is not None else None, out_w=ow if y is not None else None,
                               in_next=iw if use_in else None, w=w, eps=1e-4, h=hh)
                assert float((x2.double().cpu().view(n, S, D) - new).abs().max()) < 1e-5 * max(1.0, float(new.abs().max())), (S, D)
                assert float((hh.double().cpu() - h).abs().max()) < tol * max(1.0, float(h.abs().max())), (S, D)
        idx = torch.tensor([3, 0, 36], dtype=torch.int32, device=dev)
        assert float((ops.stream_sums(x, S, idx).double().cpu() - X[[3, 0, 36]].sum(1)).abs().max()) < 1e-5
        assert float((ops.stream_sums(x, S).double().cpu() - X.sum(1)).abs().max()) < 1e-5
    for G, gs, col, ldo in ((3, 24, 8, 96), (4, 10, 3, 50), (2, 64, 16, 160)):
        o, gate, w = torch.randn(n, G * gs, device=dev), torch.randn(n, G * gs + 4, device=dev), torch.randn(gs, device=dev)
        out = torch.full((n, ldo), 7.0, device=dev)
        ops.group_norm_gate(o, w, gate, 4, ops.ACT_X_LOGISTIC, seq, out, 1e-4, G, gs, col)
        v, z = o.double().cpu().view(n, G, gs), gate.double().cpu()[:, 4:]
        want = (v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-4) * w.double().cpu()).reshape(n, -1) * z * torch.sigmoid(z)
        want[5] = 0.0
        assert float((out[:, col:col + G * gs].double().cpu() - want).abs().max()) < 2e-5 * float(want.abs().max())
        assert float((out[:, :col] - 7).abs().max()) == 0.0 and float((out[:, col + G * gs:] - 7).abs().max()) == 0.0


def test_the_bias_epilogue_of_every_product():
    """act(x . W^T + b) with the erf-form GELU and without an activation: the few-rows kernel, the tcgen05 kernel in both
    orientations, on single SMs and on pairs of SMs, the plain kernel in both types; output columns that are no multiple of a
    tile; against float64."""
    from hos_b200 import ops
    from hos_b200.parts import gemm_tc, linear
    dev = "cuda"
    torch.manual_seed(9)
    for k, f in ((256, 384), (264, 200), (320, 331)):
        w = (torch.randn(f, k, device=dev) * 0.1).to(torch.bfloat16)
        b = torch.randn(f, device=dev)
        for m in (1, 5, 24, 40, 100, 300, 1100):
            x = torch.randn(m, k, device=dev).to(torch.bfloat16)
            z = x.double().cpu() @ w.double().cpu().T + b.double().cpu()
            for act in ("gelu_erf", "none"):
                want = 0.5 * z * (1.0 + torch.erf(z / 2 ** 0.5)) if act == "gelu_erf" else z
                size = max(1.0, float(want.abs().max()))

                def run(xx, ww):
                    return linear.matmul(xx, ww, epilogue=ops.EPI_BIAS, act=ops.BIAS_ACTIVATIONS[act], bias=b).double().cpu()
                got = run(x, w)
                assert float((got - want).abs().max()) < 8e-3 * size, f"{m} rows, {act}"
                if m == 300:
                    gemm_tc.set_pair_min_rows(0)
                    try:
                        assert float((run(x, w) - want).abs().max()) < 8e-3 * size, "single SMs"
                    finally:
                        gemm_tc.set_pair_min_rows(gemm_tc.SWAP_MAX_ROWS + 1)
                linear.force_plain(True)
                try:
                    assert float((run(x, w) - want).abs().max()) < 8e-3 * size
                    assert float((run(x.float(), w.float()) - want).abs().max()) < 1e-5 * size
                finally:
                    linear.force_plain(False)


def test_attention_into_columns_of_a_wider_row():
    """A convolution on q, k and v, the query factor, an output factor and an output that starts in the middle of a row:
    the FMA kernel with one share and several, the tensor-core kernels for many rows and for single tokens, against
    float64 on the cache as stored."""
    from hos_b200 import ops
    from hos_b200.cache.kv import KVGroup
    from hos_b200.parts.base import KVNeed, StepInfo
    dev = "cuda"
    torch.manual_seed(8)
    H, G, kd, vd, taps, T, scale, factor = 4, 2, 64, 128, 3, 200, 0.12, 0.7
    c = H * kd + G * (kd + vd)
    w, bias = torch.randn(taps, c, device=dev) * 0.5, torch.randn(c, device=dev) * 0.3
    proj = torch.randn(T, c + 12, device=dev) * 0.7
    U = proj.double().cpu()[:, 4:4 + c] + bias.double().cpu()
    pad = torch.cat([torch.zeros(taps - 1, c, dtype=torch.float64), U])
    Y = torch.stack([(pad[t:t + taps] * w.double().cpu()).sum(0) for t in range(T)])
    fac = torch.tensor([1.0 + 0.4 * np.log((p + 1) // 50 + 1) for p in range(T)], dtype=torch.float64)
    Q = Y[:, :H * kd].view(T, H, kd) * fac[:, None, None]
    K, V = Y[:, H * kd:(H + G) * kd].view(T, G, kd), Y[:, (H + G) * kd:].view(T, G, vd)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    sink = torch.zeros(H, device=dev)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        group = KVGroup(KVNeed(G, kd, None, False, vd), 1, 8, 2, 512, dtype, torch.device(dev))
        group.open_slot(1)
        group.grow(1, T)
        group.flush()
        cache = group.view(0)
        step = StepInfo(T, 1, None, i32(list(range(T))), i32([0] * T), i32([0, T]), i32([1]), i32([T]), True, False, T, T)
        q = torch.empty(T, H, kd, device=dev)
        kept = torch.randn(2, taps - 1, c, device=dev)
        ops.qkv_conv_store(proj, 4, bias, w, kept, step, q, cache, H, G, kd, vd, False, (0.4, 50))
        ops.conv_keep(proj, taps, kept, step, c, 4, bias)
        assert float((q.double().cpu() - Q).abs().max()) < 1e-5
        assert float((kept[1].double().cpu() - U[-(taps - 1):]).abs().max()) < 1e-6
        want = torch.zeros(T, H, vd, dtype=torch.float64)
        for t in range(T):
            for h in range(H):
                e = torch.exp(K[:t + 1, h // 2] @ Q[t, h] * scale)
                want[t, h] = factor * (e @ V[:t + 1, h // 2]) / (1.0 + e.sum())
        want = want.reshape(T, H * vd)
        runs = [lambda o: ops.gated_attn(q, cache, sink, None, 0, step, o, scale, 0, 0, 1, out_col=16, out_scale=factor),
                lambda o: ops.gated_attn(q, cache, sink, None, 0, step, o, scale, 0, 0, 3, out_col=16, out_scale=factor)]
        if dtype == torch.bfloat16:
            runs.append(lambda o: ops.gated_attn_mma(q, cache, sink, None, 0, step, o, scale, 0, 0, 5, out_col=16, out_scale=factor))
        for run in runs:
            out = torch.full((T, 16 + H * vd + 24), 9.0, device=dev, dtype=dtype)
            run(out)
            assert float((out[:, 16:16 + H * vd].double().cpu() - want).abs().max()) < tol * float(want.abs().max())
            assert float((out[:, :16] - 9).abs().max()) == 0.0 and float((out[:, 16 + H * vd:] - 9).abs().max()) == 0.0
        # the last token again, alone, from the kept inputs of the ones before it: the same query, and the kernels for it
        kept[1] = U[-taps:-1].float().to(dev)
        one = StepInfo(1, 1, None, i32([T - 1]), i32([0]), i32([0, 1]), i32([1]), i32([T]), False, True, 1, T)
        q1 = torch.empty(1, H, kd, device=dev)
        ops.qkv_conv_store(proj[T - 1:].contiguous(), 4, bias, w, kept, one, q1, cache, H, G, kd, vd, True, (0.4, 50))
        assert float((q1.double().cpu() - Q[-1:]).abs().max()) < 1e-5
        assert float((kept[1].double().cpu() - U[-(taps - 1):]).abs().max()) < 1e-6
        for shares in (1, 3):
            out = torch.full((1, 16 + H * vd + 24), 9.0, device=dev, dtype=dtype)
            if dtype == torch.bfloat16:
                assert ops.gated_attn_mma_decode(q1, cache, sink, None, 0, one, out, scale, 0, 0, shares, out_col=16, out_scale=factor)
            else:
                ops.gated_attn(q1, cache, sink, None, 0, one, out, scale, 0, 0, shares, out_col=16, out_scale=factor)
            assert float((out[:, 16:16 + H * vd].double().cpu() - want[-1:]).abs().max()) < tol * float(want.abs().max())
            assert float((out[:, :16] - 9).abs().max()) == 0.0 and float((out[:, 16 + H * vd:] - 9).abs().max()) == 0.0


@pytest.mark.parametrize("H, G, d, vd", [(3, 3, 16, 20), (4, 2, 64, 48), (2, 1, 200, 8), (1, 1, 7, 5), (1, 1, 300, 2)])
def test_a_scan_in_segments_gives_what_a_whole_walk_gives(H, G, d, vd):
    """Long sequences of the decay rule (decays and factors per token, or constants) and of the channel rule are walked in
    segments side by side: the same read-outs and states as the whole walk, for sequences that start and that go on,
    some of them shorter than a segment, with decays near one and decays that vanish within a segment."""
    from hos_b200 import ops
    dev = "cuda"
    torch.manual_seed(5)
    lens, starts = [1, 700, 65, 401], [0, 0, 12, 7]
    step, cu = _ragged(dev, lens, starts, [2, 0, 3, 1])
    n = sum(lens) + 1
    assert ops.mixers().fn("hos_state_scan_segment")(len(lens), H, d, vd, max(lens), 0) > 0, "these sizes are not walked in segments"
    for kind in ("token", "constant", "channel"):
        channel, g_heads = kind == "channel", H if kind == "channel" else G
        ld = -(-(2 * g_heads * d + H * vd + 3) // 4) * 4
        rows = torch.randn(n, ld, device=dev) * 0.3
        shape = {"token": (n, H), "constant": (H,), "channel": (n, H * d)}[kind]
        g = 1.0 - torch.rand(shape, device=dev) * 0.02
        if kind != "constant":
            g[::97] = 1e-3
            g[300:340] = 1e-12           # a product of these is below what 32 bits hold
        f = torch.rand(n, H, device=dev) + 0.3 if kind == "token" else None
        state = torch.randn(4, H, vd, d, device=dev)
        outs = []
        for on in (True, False):
            ops.segmented_scans = on
            try:
                kept, out = state.clone(), torch.zeros(n, H * vd, device=dev)
                ops.state_scan(rows, 0, g_heads * d, 2 * g_heads * d, False, g, kind != "constant", None, kept, step, out, H, g_heads, d, vd,
                               v_factor=f, channel_g=channel, o_mult=0.5)
                outs.append((out, kept))
            finally:
                ops.segmented_scans = True
        for a, b in zip(*outs):
            assert float((a - b).abs().max()) < 1e-5 * float(b.abs().max()), kind


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_convolution_before_norms_and_a_rotation(dtype):
    """The attention mixer with a convolution and what may follow it (a norm per head or over the projection, a rotation):
    the same as the mixer without a convolution on rows that were convolved outside."""
    from hos_b200.cache.kv import KVGroup
    from hos_b200.config.base import PartSpec
    from hos_b200.parts.base import CallStore, Runtime, StepInfo
    from hos_b200.registry import part_impl
    dev, dt = "cuda", {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    torch.manual_seed(3)
    H, G, kd, vd, width, T, taps = 4, 2, 16, 12, 24, 90, 3
    c = H * kd + G * (kd + vd)
    for norm, rot in (("head", True), ("whole", False), (False, True)):
        base = {"width": width, "n_heads": H, "n_kv_heads": G, "dim": kd, "vdim": vd, "scale": 0.3, "bias": True, "qk_norm": norm,
                "position": PartSpec("rotary", {"theta": 100.0, "rotary_dim": 8, "style": "interleaved"}) if rot else None}
        names = {r: r for r in ("q", "k", "v", "o", "q_bias", "k_bias", "v_bias", "q_norm", "k_norm", "q_conv", "k_conv", "v_conv")}
        outs = []
        rt = Runtime(torch.device(dev), dt)
        with_conv = part_impl("mixer", "gated_softmax_attention")(PartSpec("gated_softmax_attention", dict(base, conv=taps), names), rt)
        plain = part_impl("mixer", "gated_softmax_attention")(PartSpec("gated_softmax_attention", dict(base, bias=False), names), rt)
        g = torch.Generator().manual_seed(1)
        tensors = {s.name: torch.randn(tuple(s.shape), generator=g).to(dev) for s in with_conv.weight_specs()}
        with_conv.bind(tensors)
        plain.bind(tensors)
        proj = torch.randn(T, c, device=dev)
        u = torch.cat([torch.zeros(taps - 1, c, device=dev), proj + with_conv.bias])
        convolved = sum(u[j:j + T] * with_conv.conv_w[j] for j in range(taps)).contiguous()
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        cuts = [(0, 50), (50, 89), (89, 90)]
        for m, rows in ((with_conv, proj), (plain, convolved)):
            group = KVGroup(m.kv_need(), 1, 4, 2, 128, dt, torch.device(dev))
            group.open_slot(1)
            group.grow(1, T)
            group.flush()
            store = CallStore(group.view(0), True, {"conv": torch.full((2, taps - 1, c), 5.0, device=dev)})
            att = torch.empty(T, H * vd, device=dev, dtype=dt)
            for a, b in cuts:
                step = StepInfo(b - a, 1, None, i32(list(range(a, b))), i32([0] * (b - a)), i32([0, b - a]), i32([1]), i32([b]), a == 0,
                                b - a == 1, b - a, b)
                m.run_heads(rows[a:b].contiguous(), 0, step, store, att[a:b], 0)
            outs.append(att.float())
        tol = 2e-5 if dtype == "float32" else 2e-2
        assert float((outs[0] - outs[1]).abs().max()) < tol * float(outs[1].abs().max()), (norm, rot)
