"""Ravutar without a GPU: the configuration's checks, the plan (arrangement, parts, run order, tensor names and shapes)
and properties of the oracle itself that the GPU tests rely on."""
import copy
import math

import pytest
import torch

from ravutar_cases import CASES, make_folder, oracle_view, row_errors, tokens


def test_the_plan_names_every_tensor_once():
    from hos_b200.model import weight_specs_for
    from hos_b200.registry import config_from_dict, plan_for
    cfg = config_from_dict(CASES["A"][0])
    plan = plan_for(cfg)
    assert [l.arrangement for l in plan.layers] == ["hyper_prenorm"] * 3 and plan.streams == 3
    assert [l.mixer.kind for l in plan.layers] == ["parallel_mixers", "state_space", "parallel_mixers"]
    assert [c.layer for c in plan.schedule] == [0, 1, 0, 1, 2] and all(c.cache_from is None for c in plan.schedule)
    sides = plan.layers[0].mixer.params["mixers"]
    assert list(sides) == ["left", "right"] and sides["left"].params["q_temp"] == {"coef": 0.4, "every": 16}
    assert sides["left"].params["out_scale"] == 0.7 and sides["right"].params["out_scale"] == 1.1
    assert plan.layers[2].feed_forward.kind == "none" and set(plan.layers[2].norms) == {"pre_mixer"}
    assert plan.final_norm.params["mult"] == 0.6 and plan.embedding.params["copies"] == 3
    names = {s.name: tuple(s.shape) for s in weight_specs_for(cfg)}
    assert names["embed"] == (211, 72) and names["head"] == (211, 72) and names["final.norm"] == (72,)
    assert names["l0.mix.left.q"] == (72, 72) and names["l0.mix.left.k"] == (24, 72) and names["l0.mix.left.v"] == (16, 72)
    assert names["l0.mix.left.q.b"] == (72,) and names["l0.mix.left.v.conv"] == (16, 4) and names["l0.mix.left.o"] == (72, 48)
    assert names["l0.mix.left.o.b"] == (72,) and names["l0.mix.right.q"] == (24, 72) and names["l0.mix.right.g"] == (40, 72)
    assert names["l0.mix.right.a1"] == (5, 72) and names["l0.mix.right.a2"] == (24, 5) and names["l0.mix.right.a2.b"] == (24,)
    assert names["l0.mix.right.norm"] == (20,) and names["l0.mix.right.o"] == (72, 40)
    assert names["l1.mix.in"] == (2 * 72 + 2 * 60 + 6, 72) and names["l1.mix.conv"] == (192, 3) and names["l1.mix.conv.b"] == (192,)
    assert names["l1.mix.D"] == (6,) and names["l1.mix.norm"] == (72,) and names["l1.mix.o"] == (72, 72)
    assert names["l0.mlp.up.b"] == (56,) and names["l0.mlp.down"] == (72, 56) and names["l1.hc2.mix"] == (3, 3)
    assert names["l2.hc1.in"] == (3,) and "l2.hc2.in" not in names and "l2.norm2" not in names and "l2.mlp.up" not in names
    assert config_from_dict(cfg.to_dict()) == cfg


def test_sizes_that_a_checkpoint_gives_need_no_configuration():
    from hos_b200.errors import MissingMetaError
    from hos_b200.model import weight_specs_for
    from hos_b200.registry import config_from_dict
    from hos_b200.weights import RandomSource
    raw = copy.deepcopy(CASES["A"][0])
    raw["layers"][0]["mixer"]["right"].pop("decay_rank")
    cfg = config_from_dict(raw)
    names = {s.name: tuple(s.shape) for s in weight_specs_for(cfg)}
    assert names["l0.mix.right.a1"] == (-1, 72) and names["l0.mix.right.a2"] == (24, -1)
    with pytest.raises(MissingMetaError):
        RandomSource(weight_specs_for(cfg), 0)


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=2), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("tau"), "tau"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(dim="x"), "dim"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0].update(type="recurrence"), "type"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c["loop"].update(stop=4), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_a_wrong_configuration_is_refused_with_the_key_named(edit, word):
    from hos_b200.errors import MissingMetaError
    from hos_b200.registry import config_from_dict
    raw = copy.deepcopy(CASES["A"][0])
    edit(raw)
    with pytest.raises(MissingMetaError) as e:
        config_from_dict(raw)
    assert word in str(e.value)


def test_only_mixers_that_say_how_stand_side_by_side():
    from hos_b200.config.base import PartSpec
    from hos_b200.errors import SpecError
    from hos_b200.parts.base import Runtime
    from hos_b200.registry import config_from_dict, part_impl, plan_for
    rt = Runtime(torch.device("cpu"), torch.bfloat16)
    plan = plan_for(config_from_dict(CASES["A"][0]))
    sides = plan.layers[0].mixer.params["mixers"]
    both = part_impl("mixer", "parallel_mixers")(PartSpec("parallel_mixers", {"mixers": sides}), rt)
    assert {s.name: s.shape for s in both.state_needs()} == {"left.conv": (3, 112), "right.S": (2, 20, 12)}
    assert both.kv_need().n_kv_heads == 1 and both.kv_need().head_dim == 24 and both.kv_need().v_head_dim == 16
    with pytest.raises(SpecError):
        part_impl("mixer", "parallel_mixers")(PartSpec("parallel_mixers", {"mixers": {"a": sides["left"], "b": plan.layers[1].mixer}}), rt)
    with pytest.raises(SpecError):
        part_impl("mixer", "parallel_mixers")(PartSpec("parallel_mixers", {"mixers": {"a": sides["left"], "b": sides["left"]}}), rt)


def test_the_oracle_feels_every_mechanism(tmp_path):
    """What the GPU tests compare with must move when a mechanism is taken away or changed a little."""
    from plain import ravutar_plain as P
    folder = make_folder(tmp_path, CASES["A"][0], CASES["A"][1], "A")
    cfg, w = oracle_view(folder)
    seq = tokens(1, 110, cfg["vocab"])
    want = P.forward(cfg, w, seq)

    def moved(edit=None, rows=slice(60, None), order=None, cfg2=None, **changed):
        got = P.forward(cfg2 or cfg, dict(w, **changed), seq, edit=edit, order=order)
        return float(row_errors(got[rows], want[rows]).median())

    def left(**kw):
        return lambda i, m: dict(m, left=dict(m["left"], **kw)) if "left" in m else m
    far = 2e-3
    assert moved(left(no_sink=True)) > far and moved(left(only_last=30)) > far
    assert moved(left(q_temp=None)) > far
    for i in (0, 2):                                        # each layer's own factor, its step one off
        t = cfg["layers"][i]["mixer"]["left"]["q_temp"]
        for d in (1, -1):
            def edit(j, m):
                return dict(m, left=dict(m["left"], q_temp=dict(t, every=t["every"] + d))) if j == i else m
            assert moved(edit) > far / 4, (i, d)
    for name in ("l0.mix.left.q", "l0.mix.left.k", "l0.mix.left.v"):
        only_now = torch.zeros_like(w[name + ".conv"])
        only_now[:, -1] = w[name + ".conv"][:, -1]
        assert moved(**{name + ".conv": only_now}) > far, name
        assert moved(**{name + ".conv": w[name + ".conv"].roll(1, 1)}) > far, name
        # a key bias alone is seen through the convolution at a sequence's start only
        assert moved(**{name + ".b": torch.zeros_like(w[name + ".b"])}, rows=slice(0, None)) > far / 8, name
    assert moved(**{"l2.mix.left.o.b": torch.zeros_like(w["l2.mix.left.o.b"])}) > far
    assert moved(lambda i, m: dict(m, left_scale=m["left_scale"] * 1.05) if "left" in m else m) > far
    assert moved(lambda i, m: dict(m, right_scale=m["right_scale"] * 1.05) if "left" in m else m) > far
    assert moved(lambda i, m: dict(m, right=dict(m["right"], tau=m["right"]["tau"] * 1.1)) if "right" in m else m) > far
    for name in ("l0.mix.right.a1", "l0.mix.right.a2.b", "l0.mix.right.g", "l2.mix.right.a2"):
        assert moved(**{name: w[name] * 0.5}) > far / 4, name
    assert moved(**{"l1.mix.conv": w["l1.mix.conv"].roll(1, 1)}) > far
    for name in ("l1.mix.conv.b", "l1.mix.dt_bias", "l1.mix.A_log", "l1.mix.D", "l1.mix.norm"):
        assert moved(**{name: torch.zeros_like(w[name])}) > far, name
    assert moved(lambda i, m: dict(m, norm_groups=2) if "norm_groups" in m else m) > far
    assert moved(lambda i, m: dict(m, groups=6, state=10) if "norm_groups" in m else m) > far      # how the columns are laid out
    for name in ("l0.mlp.up.b", "l0.mlp.down.b"):
        assert moved(**{name: torch.zeros_like(w[name])}) > far, name
    for name in ("l0.hc1.mix", "l1.hc2.mix", "l2.hc1.mix"):
        assert moved(**{name: w[name].T}) > far, name        # [from, to]
    for name in ("l0.hc2.in", "l1.hc1.out", "l2.hc1.in"):
        assert moved(**{name: w[name].flip(0)}) > far / 4, name
    assert moved(order=[0, 1, 2]) > far and moved(order=[0, 0, 1, 1, 2]) > far                     # the loop
    assert moved(cfg2=dict(cfg, logit_scale=0.7)) > far
    # prefix property: a position's logits do not depend on later tokens
    assert float(row_errors(P.forward(cfg, w, seq[:60]), want[:60]).max()) < 1e-12


def test_pieces_of_the_oracle_against_closed_forms():
    """The recurrences unrolled by hand on three tokens, the query factor's steps, the sink on one key."""
    from plain import ravutar_plain as P
    assert P.query_factor(None, 50) == 1.0
    t = {"coef": 0.5, "every": 4}
    assert P.query_factor(t, 2) == 1.0 and abs(P.query_factor(t, 3) - (1 + 0.5 * math.log(2))) < 1e-15
    assert P.query_factor(t, 6) == P.query_factor(t, 3) and abs(P.query_factor(t, 7) - (1 + 0.5 * math.log(3))) < 1e-15
    u = torch.randn(4, 2, dtype=torch.float64)
    wc = torch.randn(2, 3, dtype=torch.float64)
    y = P.short_conv(u, wc)
    assert torch.allclose(y[0], wc[:, 2] * u[0]) and torch.allclose(y[1], wc[:, 2] * u[1] + wc[:, 1] * u[0])
    assert torch.allclose(y[3], wc[:, 2] * u[3] + wc[:, 1] * u[2] + wc[:, 0] * u[1])
    # one head of one number each, attention of one key: v e^s / (1 + e^s)
    one = torch.ones(1, 1, dtype=torch.float64)
    w = {"q": 2 * one, "k": 3 * one, "v": 5 * one, "o": one, "q.b": one[0], "k.b": one[0], "v.b": one[0], "o.b": 7 * one[0],
         "q.conv": one, "k.conv": one, "v.conv": one}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.1, "conv": 1}
    s = (2 + 1) * (3 + 1) * 0.1
    assert abs(float(P.softmax_branch(m, w, "", one)) - (6 * math.exp(s) / (1 + math.exp(s)) + 7)) < 1e-12
    # the decay: logistic(z)^(1/tau)
    d = P.channel_decay({"heads": 1, "dim": 1, "tau": 4.0}, {"a1": 2 * one, "a2": 0.5 * one, "a2.b": 0.25 * one[0]}, "", one)
    assert abs(float(d) - (1 / (1 + math.exp(-1.25))) ** 0.25) < 1e-12


def test_a_constant_on_a_norm_is_folded_into_its_weight():
    from hos_b200.config.base import PartSpec
    from hos_b200.parts.base import Runtime
    from hos_b200.parts.norm import RMSNorm
    w = torch.randn(12).to(torch.bfloat16)
    rt = Runtime(torch.device("cpu"), torch.bfloat16)
    n = RMSNorm(PartSpec("rmsnorm", {"width": 12, "eps": 1e-6, "mult": 0.25}, {"weight": "w"}), rt)
    n.bind({"w": w})
    assert torch.equal(n.weight.double(), w.double() * 0.25)
    g = RMSNorm(PartSpec("rmsnorm", {"width": 12, "eps": 1e-6, "add_one": True, "mult": 3.0}, {"weight": "w"}), rt)
    g.bind({"w": w})
    assert float(((g.weight.double() + 1.0) - (w.double() + 1.0) * 3.0).abs().max()) < 1e-6
