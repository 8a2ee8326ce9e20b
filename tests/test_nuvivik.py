"""Nuvivik without a GPU: the configuration's checks, the plan (arrangement, parts, run order, tensor names and shapes)
and properties of the oracle itself that the GPU tests rely on."""
import copy
import math

import pytest
import torch

from nuvivik_cases import CASES, make_folder, oracle_view, row_errors, tokens


def test_the_plan_names_every_tensor_once():
    from hos_b200.model import weight_specs_for
    from hos_b200.registry import config_from_dict, plan_for
    cfg = config_from_dict(CASES["A"][0])
    plan = plan_for(cfg)
    assert [l.arrangement for l in plan.layers] == ["branch_norm"] * 4
    assert [l.mixer.kind for l in plan.layers] == ["latent_attention", "gated_softmax_attention"] * 2
    assert [l.feed_forward.kind for l in plan.layers] == ["dense_mlp", "routed_experts", "none", "routed_experts"]
    assert [c.cache_from for c in plan.schedule] == [None] * 4
    assert [l.mixer.params["window"] for l in plan.layers] == [33, 70, 64, None]
    assert plan.layers[0].mixer.params["q_rank"] == 20 and plan.layers[0].mixer.params["sink"]
    pos = plan.layers[1].mixer.params["position"].params
    assert pos["style"] == "rotate_half" and pos["rotary_dim"] == 8
    assert pos["scaling"] == {"kind": "bands", "factor": 8.0, "low": 1.0, "high": 4.0, "original": 100.0}
    assert plan.layers[0].mixer.params["position"].params["scaling"] is None
    assert plan.layers[1].mixer.params["softcap"] == 4.0 and plan.layers[1].mixer.params["qk_norm"] == "unit"
    assert plan.layers[1].feed_forward.params["groups"] == {"count": 3, "keep": 2}
    assert plan.layers[3].feed_forward.params["groups"] is None
    assert plan.final_norm.params["mult"] == 0.7 and plan.head.params["softcap"] == 1.5 and plan.embedding.params["scale"] == 3.0
    assert set(plan.layers[2].norms) == {"post_mixer"} and set(plan.layers[0].norms) == {"post_mixer", "post_ffn"}
    names = {s.name: tuple(s.shape) for s in weight_specs_for(cfg)}
    assert names["embed"] == (211, 72) and names["head"] == (211, 72) and names["final.norm"] == (72,)
    assert names["l0.mix.dq"] == (20, 72) and names["l0.mix.dq.norm"] == (20,) and names["l0.mix.uq"] == (72, 20)
    assert names["l0.mix.dkv"] == (48, 72) and names["l0.mix.dkv.norm"] == (40,) and names["l0.mix.sink"] == (3,)
    assert names["l0.mix.uk"] == (48, 40) and names["l0.mix.uv"] == (72, 40) and names["l0.mix.o"] == (72, 72)
    assert names["l1.mix.q"] == (72, 72) and names["l1.mix.k"] == (24, 72) and names["l1.mix.v"] == (16, 72)
    assert names["l1.mix.q.b"] == (72,) and names["l1.mix.k.b"] == (24,) and names["l1.mix.v.b"] == (16,)
    assert names["l1.mix.o"] == (72, 48) and "l1.mix.sink" not in names and "l1.mix.q.norm" not in names
    assert names["l0.mlp.up"] == (56, 72) and names["l0.mlp.down"] == (72, 56) and "l0.mlp.up.b" not in names
    assert names["l1.mlp.router"] == (6, 72) and names["l1.mlp.e5.up"] == (40, 72) and names["l1.mlp.e0.down"] == (72, 40)
    assert "l1.mlp.e0.gate" not in names and "l2.norm2" not in names and "l2.mlp.up" not in names and "l0.mix.q" not in names
    assert names["l0.norm1"] == (72,) and names["l3.norm2"] == (72,)
    assert config_from_dict(cfg.to_dict()) == cfg


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=0), "vdim"),
    (lambda c: c["layers"][0].update(type="recurrence"), "type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c.update(logit_softcap=-2.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.pop("layers"), "layers"),
])
def test_a_wrong_configuration_is_refused_with_the_key_named(edit, word):
    from hos_b200.errors import MissingMetaError
    from hos_b200.registry import config_from_dict
    raw = copy.deepcopy(CASES["A"][0])
    edit(raw)
    with pytest.raises(MissingMetaError) as e:
        config_from_dict(raw)
    assert word in str(e.value)


def test_parts_refuse_what_they_cannot_do():
    from hos_b200.config.base import PartSpec
    from hos_b200.errors import SpecError
    from hos_b200.parts.base import Runtime
    from hos_b200.registry import part_impl
    rt = Runtime(torch.device("cpu"), torch.float32)
    base = {"width": 8, "inner": 8, "experts": 6, "top": 2, "activation": "relu_square", "scoring": "logistic"}
    part_impl("feed_forward", "routed_experts")(PartSpec("routed_experts", dict(base, groups={"count": 3, "keep": 1})), rt)
    for bad in ({"groups": {"count": 4, "keep": 1}}, {"groups": {"count": 3, "keep": 4}}, {"groups": {"count": 6, "keep": 1}},
                {"activation": "cube"}):
        with pytest.raises(SpecError):
            part_impl("feed_forward", "routed_experts")(PartSpec("routed_experts", dict(base, **bad)), rt)
    ramp = PartSpec("rotary", {"theta": 100.0, "rotary_dim": 4, "scaling": {"factor": 2.0, "original": 10, "fast": 4, "slow": 1}})
    with pytest.raises(SpecError):           # a ramp's cosines are multiplied: a norm before it is not the same after it
        part_impl("mixer", "gated_softmax_attention")(
            PartSpec("gated_softmax_attention", {"width": 8, "n_heads": 1, "n_kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0,
                                                 "qk_norm": "unit", "position": ramp}), rt)
    with pytest.raises(SpecError):
        part_impl("position", "rotary")(PartSpec("rotary", {"theta": 9.0, "rotary_dim": 4, "scaling": {"kind": "bends"}}), rt)


def test_banded_frequencies_of_the_part_and_of_the_oracle():
    """Fast pairs as they are, slow ones divided by the factor, the ones between on the line that joins the two; a band of no
    width; the same numbers as the oracle's."""
    from hos_b200.config.base import PartSpec
    from hos_b200.parts.base import Runtime
    from hos_b200.registry import part_impl
    from plain import nuvivik_plain as P
    rt = Runtime(torch.device("cpu"), torch.float32)
    for dims, base, bands in ((8, 100.0, (8.0, 1.0, 4.0, 100.0)), (64, 10000.0, (4.0, 1.0, 4.0, 512.0)), (24, 77.0, (2.0, 0.3, 0.3, 30.0))):
        sc = dict(zip(("factor", "low", "high", "original"), bands))
        part = part_impl("position", "rotary")(PartSpec("rotary", {"theta": base, "rotary_dim": dims, "style": "rotate_half",
                                                                   "scaling": dict(sc, kind="bands")}), rt)
        assert part.magnitude == 1.0
        want = P.frequencies({"dims": dims, "base": base, "scaling": sc})
        got = part.kernel_args()[0].double()
        assert float((got / torch.tensor(want, dtype=torch.float64) - 1).abs().max()) < 1e-7
        plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        ratio = [a / b for a, b in zip(want, plain)]
        assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / bands[0]) < 1e-12 and all(1 / bands[0] - 1e-12 <= r <= 1.0 for r in ratio)
        if bands[1] != bands[2]:
            assert any(1 / bands[0] + 1e-3 < r < 0.999 for r in ratio)          # a pair in between
    # one pair by hand: half way between low and high
    sc = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 2.0 * (2 * math.pi)}
    (f,) = P.frequencies({"dims": 2, "base": 5.0, "scaling": sc})               # f = 1, original / wavelength = 2
    assert abs(f - (0.5 / 4 + 0.5)) < 1e-12


def test_the_oracle_feels_every_mechanism(tmp_path):
    """What the GPU tests compare with must move when a mechanism is taken away or shifted by one."""
    from plain import nuvivik_plain as P
    folder = make_folder(tmp_path, CASES["A"][0], CASES["A"][1], "A")
    cfg, w = oracle_view(folder)
    seq = tokens(1, 110, cfg["vocab"])
    want = P.forward(cfg, w, seq)

    def moved(edit=None, cfg2=None, rows=slice(80, None), **changed):
        got = P.forward(cfg2 or cfg, dict(w, **changed), seq, edit=edit)
        return float(row_errors(got[rows], want[rows]).median())

    def change(i, **kw):
        return lambda j, m: dict(m, **kw) if j == i else m
    far = 2e-3
    for i in (0, 1, 2):
        for d in (1, -1):
            size = cfg["layers"][i]["mixer"]["mask"]["size"]
            assert moved(change(i, mask={"size": size + d})) > far / 4, (i, d)
    for i in (1, 3):
        assert moved(change(i, softcap=None)) > far, i
        for n in ("q.b", "k.b", "v.b"):
            assert moved(**{f"l{i}.mix.{n}": torch.zeros_like(w[f"l{i}.mix.{n}"])}) > far / 4, (i, n)
    for i in (0, 2):
        assert moved(**{f"l{i}.mix.sink": w[f"l{i}.mix.sink"] - 50.0}) > far, i
        for n in ("dq.norm", "dkv.norm"):
            assert moved(**{f"l{i}.mix.{n}": torch.ones_like(w[f"l{i}.mix.{n}"])}) > far, (i, n)
    rot1 = cfg["layers"][1]["mixer"]["rot"]
    assert moved(change(1, rot={k: v for k, v in rot1.items() if k != "scaling"})) > far
    for key, v in (("factor", 4.0), ("low", 0.5), ("high", 8.0), ("original", 60)):
        assert moved(change(1, rot=dict(rot1, scaling=dict(rot1["scaling"], **{key: v})))) > far / 8, key
    for i in range(4):
        rot = cfg["layers"][i]["mixer"]["rot"]
        assert moved(change(i, rot=dict(rot, base=rot["base"] * 2))) > far / 4, i
        assert moved(change(i, scale=cfg["layers"][i]["mixer"]["scale"] * 1.1)) > far / 2, i
        assert moved(**{f"l{i}.norm1": w[f"l{i}.norm1"] * 1.05}) > far, i
    for key in ("logit_scale", "logit_softcap"):
        assert moved(cfg2=dict(cfg, **{key: cfg[key] * 1.1})) > far, key
    assert moved(cfg2=dict(cfg, embedding={"scale": 3.3})) > far
    free = copy.deepcopy(cfg)
    free["layers"][1]["mlp"]["router"].pop("groups")                    # the groups rule some tokens' choice
    assert float((row_errors(P.forward(free, w, seq), want) > far).double().mean()) > 0.2
    # a query and a key of another length is the same query and key
    for n in ("q", "k"):
        t = dict(w, **{f"l1.mix.{n}": w[f"l1.mix.{n}"] * 2, f"l1.mix.{n}.b": w[f"l1.mix.{n}.b"] * 2})
        assert float(row_errors(P.forward(cfg, t, seq), want).max()) < 1e-4
    # prefix property: a position's logits do not depend on later tokens
    assert float(row_errors(P.forward(cfg, w, seq[:60]), want[:60]).max()) < 1e-12


def test_the_choice_of_experts_by_groups():
    from plain import nuvivik_plain as P
    s = torch.tensor([0.875, 0.125, 0.125, 0.625, 0.5, 0.375, 0.75, 0.25, 0.1875])          # three groups: sums 1, 1.125, 1
    assert P.choose({"top": 3}, s) == [0, 6, 3]
    assert P.choose({"top": 2, "groups": {"count": 3, "keep": 1}}, s) == [3, 4]
    assert P.choose({"top": 3, "groups": {"count": 3, "keep": 2}}, s) == [0, 3, 4]        # equal groups: the first
    assert P.choose({"top": 2, "groups": {"count": 9, "keep": 3}}, s) == [0, 6]           # groups of one
    # the weights are the scores as they are
    w = {"router": torch.tensor([[2.0], [0.0]], dtype=torch.float64)}
    for e in range(2):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.tensor([[3.0 + e]], dtype=torch.float64), torch.ones(1, 1, dtype=torch.float64)
    y = P.routed_ff({"router": {"experts": 2, "top": 2}}, w, "", torch.ones(1, 1, dtype=torch.float64))
    assert abs(float(y) - (9.0 / (1 + math.exp(-2.0)) + 16.0 * 0.5)) < 1e-12
    y = P.routed_ff({"router": {"experts": 2, "top": 2}}, w, "", -torch.ones(1, 1, dtype=torch.float64))
    assert float(y) == 0.0                                                     # the square of relu
