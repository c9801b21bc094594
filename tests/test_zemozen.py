"""Zemozen without a GPU: configuration and registry, constants and layout of its layers, the oracle's sensitivity to the faults
the GPU tests look for, generation by the scheduler and the servers over the oracle."""
import copy
import json

import pytest
import torch
import zemozen_reference as zr
from gidisun_cases import OracleRuntime
from zemozen_cases import BEACON, FULL, attention, beacon_tensors, clear_routes, config, moe, parallel, tensors, tokens

from pocketllm_b200.models import mixer_layers as ml
from pocketllm_b200.models import registry
from pocketllm_b200.models import zemozen as zm
from pocketllm_b200.runtime.batching import BatchEngine
from pocketllm_b200.runtime.mixer_runtime import plan_portions
from pocketllm_b200.server.engine import SamplingParams, ServingEngine

SMALL = config([parallel(moe(experts=3, identity=1, top=2)), attention(window=7), attention(window=9)], width=40)


def test_config_registry_and_checkpoint_folder(tmp_path):
    c = zm.ZemozenConfig.from_dict(FULL)
    assert (c.residual_mult, c.first_v_mix()) == (0.45, 1) and c.layers[3].identity == 0 and c.layers[2].mlp is None
    t = tensors(FULL)
    assert set(t) == set(zm.tensor_plan(c)) and t["l0.mlp.router"].shape == (7, 88) and t["l3.mix.right.in"].shape == (4 * 33 * 2 + 2 * 70 + 4, 88)
    assert "l1.mix.vmix" in t and "l2.mix.vmix" not in t and t["l1.mix.vmix"].shape == ()
    zm.save_checkpoint(tmp_path, c, t)
    assert json.loads((tmp_path / "config.json").read_text()) == FULL
    assert zm.ZemozenConfig.load(tmp_path) == c
    assert registry.folder_architecture(tmp_path) == "Zemozen" and "Zemozen" in registry.architectures()
    back = zm.load_tensors(tmp_path)
    assert all(torch.equal(back[k], t[k]) for k in t)
    from pocketllm_b200.server import openai as oa
    assert oa.detect_model_kind(str(tmp_path)) == "mixer"


def changed(layer, *path_value):
    L = copy.deepcopy(layer)
    *path, last, value = path_value
    m = L["mixer"]
    for k in path:
        m = m[k]
    m[last] = value
    return dict(layers=[L])


@pytest.mark.parametrize("bad", [
    dict(layers=[{"type": "retention", "mixer": {}, "mlp": None}]),
    dict(layers=[{"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8}, "mlp": None}]),
    dict(layers=[{"type": "parallel", "mixer": {"left": parallel()["mixer"]["left"]}, "mlp": None}]),
    dict(layers=[attention(rot=5)]), dict(layers=[attention(dim=8, rot=10)]), dict(layers=[attention(heads=3, kv=2)]),
    dict(layers=[attention(factor=-1.0)]),
    dict(layers=[attention(), attention(vdim=20)]),
    dict(layers=[parallel(heads_=4, groups=3)]), dict(layers=[parallel(heads_=3, vdim=5, groups=1, parts=2)]), dict(layers=[parallel(conv=0)]),
    dict(layers=[parallel(cap=0.0)]), changed(parallel(), "left", "kv_heads", 3), changed(attention(), "mask", "size", 0),
    dict(layers=[attention(moe(experts=3, identity=1, top=5))]), dict(layers=[attention(moe(experts=0))]),
    dict(layers=[attention({"kind": "dense", "ff": 8})]),
    dict(architecture="Pezarax"),
])
def test_config_refuses_what_it_does_not_know(bad):
    with pytest.raises(ValueError):
        zm.ZemozenConfig.from_dict(FULL | bad)


def test_missing_and_misshapen_tensors_are_refused():
    c, t = zm.ZemozenConfig.from_dict(FULL), tensors(FULL)
    with pytest.raises(KeyError, match="l0.mix.right.dt_bias"):
        zm.build_model(c, {k: v for k, v in t.items() if k != "l0.mix.right.dt_bias"}, device="cpu")
    with pytest.raises(ValueError, match="l1.mlp.e3.gate"):
        zm.build_model(c, t | {"l1.mlp.e3.gate": t["l1.mlp.e3.gate"][:-1]}, device="cpu")


def test_layers_of_the_model():
    """Constants, columns and memory of the layers."""
    c, t = zm.ZemozenConfig.from_dict(FULL), tensors(FULL)
    m = zm.build_model(c, t, device="cpu", slots=3, pages=5, dtype=torch.bfloat16)
    assert [getattr(L.mixer, "desc", {}).get("v_mix", 0) for L in m.layers] == [0, 1, 0, 0, 2]
    assert m.layers[4].mixer.desc["mix"] == pytest.approx(float(t["l4.mix.vmix"])) and (m.residual_scale, m.embed_scale) == (0.45, 2.5)
    p = m.layers[3].mixer
    left, right = p.left, p.right
    assert left.desc["neighbours"] == 1 and left.desc["window"] == 65 and left.desc["gate"] == -1 and left.desc["cap"] == 2.5
    assert left.const["sink"].tolist() == [0.0] * 4 and left.desc["post"] == 1.0 and m.layers[0].mixer.left.desc["post"] == pytest.approx(0.7)
    assert left.const["freq"].tolist() == pytest.approx([700.0 ** (-2 * i / 40) / 2.0 for i in range(20)])
    a = p.proj.at
    assert (left.desc["oq"], left.desc["ok"], left.desc["ov"]) == (0, 4 * 40, 5 * 40) and a["right"] == 5 * 40 + 132
    assert (right.desc["og"], right.desc["ov"], right.desc["odt"]) == (a["right"], a["right"] + 132, a["right"] + 2 * 132 + 140)
    assert right.S.shape == (3, 4, 70, 33) and right.ring.shape == (3, 2, 132 + 140) and left.cache.shape == (5, 64, 40 + 136)
    assert p.split == 520 and torch.equal(p.out.w[:88, 520:520 + 132], t["l3.mix.right.o"]) and (p.out.w[:, 652:] == 0).all()
    assert torch.allclose(right.norm, t["l3.mix.right.norm"].float() * 0.4)
    assert m.layers[1].mixer.desc["gate"] == m.layers[1].mixer.proj.at["g"] and m.layers[1].mixer.desc["neighbours"] == 0
    e = m.layers[0].mlp
    assert e.gated and (e.route.experts, e.route.identity, e.route.outputs) == (5, 2, 7) and e.up.shape == (5, 256, 128)
    assert torch.equal(e.up[2, :36, :88], t["l0.mlp.e2.gate"]) and torch.equal(e.up[2, 128:164, :88], t["l0.mlp.e2.up"])


def test_slowed_down_rotations():
    f, mag = ml.rotary_frequencies(8, 100.0, {"factor": 5.0})
    assert mag == 1.0 and f.tolist() == pytest.approx([100.0 ** (-i / 4) / 5 for i in range(4)])


def test_portions_know_the_tokens_after_a_row():
    p = plan_portions([3, 1, 10], [5, 0, 64], [0, 2, 1], windows=[])
    assert p["behind"].tolist() == [2, 1, 0, 0] + list(range(9, -1, -1))
    p = plan_portions([300, 2, 128, 129], [0, 5, 64, 1], [0, 2, 1, 3], windows=[])
    assert p["tile0"] == [0, 3, 4] and [t[:3] for t in p["tiles"]] == [(0, 128, 0), (128, 128, 0), (256, 44, 0), (302, 128, 1), (430, 128, 2), (558, 1, 2)]


@pytest.mark.parametrize("fault", ["window", "window_parallel", "sink", "cap", "pairs", "head_norm", "v_mix", "gate", "skip", "groups", "residual",
                                   "identity", "correction"])
def test_oracle_notices_faults(fault):
    """The tests' weights make each of these faults visible."""
    place = slice(None)
    if fault.startswith("window"):
        cfg = config([parallel(left={"window": 37}, cap=30.0) if "parallel" in fault else attention(window=29)])
        t = beacon_tensors(cfg)
        seq = tokens(60, cfg["vocab"], 3, low=1)
        seq[20] = BEACON
        place = slice(57, 58) if "parallel" in fault else slice(49, 50)      # the first token that does not see it any more
        fault = "window"
    else:
        cfg = config(SMALL["layers"])
        t = tensors(cfg)
        if fault in ("identity", "correction"):
            t = clear_routes(cfg, t)
        seq = tokens(14, cfg["vocab"], 3)
    good = zr.PlainModel(cfg, t).logits(seq)
    zr.MUTATE.add(fault)
    try:
        bad = zr.PlainModel(cfg, t).logits(seq)
    finally:
        zr.MUTATE.clear()
    d = (good - bad).pow(2).mean(-1).sqrt() / good.std()
    assert d[place].max() > 0.05


@pytest.mark.parametrize("cfg,last", [(config([attention(window=29)]), 48), (config([parallel(left={"window": 37}, cap=30.0)]), 56)])
def test_oracle_sees_keys_to_the_end_of_their_window(cfg, last):
    t = beacon_tensors(cfg)
    if cfg["layers"][0]["type"] == "parallel":      # the recurrence remembers the token as well
        t["l0.mix.right.o"] = torch.zeros_like(t["l0.mix.right.o"])
    seq = tokens(70, cfg["vocab"], 3, low=1)
    seq[20] = BEACON
    a, b = (zr.PlainModel(cfg, t).logits(s) for s in (seq, seq[:20] + [5] + seq[21:]))
    d = (a - b).pow(2).mean(-1).sqrt() / a.std()
    assert d[last] > 0.1 and d[last + 1] < 1e-9


def test_routes_of_the_test_weights_are_clear():
    t = clear_routes(FULL, tensors(FULL))
    m = zr.PlainModel(FULL, t)
    gaps, seen, turned = [], set(), 0
    plain = zr.route

    def watch(w, cfg, h):
        nonlocal turned
        s = torch.softmax(w["router"] @ h, 0)
        c, k = (s + w["correction"]).sort(descending=True).values, cfg["router"]["top"]
        if k < len(c):
            gaps.append(float(c[k - 1] - c[k]))
        out = plain(w, cfg, h)
        seen.update((len(s), e) for e, _ in out)
        turned += {e for e, _ in out} != set(torch.topk(s, k).indices.tolist())
        return out
    zr.route = watch
    try:
        m.logits(tokens(25, FULL["vocab"], 1))
    finally:
        zr.route = plain
    assert min(gaps) > 2e-3 and turned > 10
    assert {(7, 5), (5, 1), (3, 2)} <= seen                           # an identity among them


def test_generation_by_the_scheduler_and_the_server():
    from pocketllm_b200.server.backends import MixerBackend
    t = tensors(SMALL)
    rt = OracleRuntime(SMALL, t, max_requests=3, pages=12, page=16, plain=zr.PlainModel)
    m = zr.PlainModel(SMALL, t)
    prompts = [tokens(n, SMALL["vocab"], n) for n in (5, 21, 1, 17)]
    eng = BatchEngine(rt, token_budget=12, burst=4)
    outs = eng.run(prompts, [SamplingParams(max_tokens=n) for n in (7, 6, 9, 3)])
    for p, o in zip(prompts, outs):
        assert o == m.generate(p, len(o))
    assert eng.stats["mixed_steps"] > 0 and rt.cache.free_pages == 12
    srv = ServingEngine(MixerBackend(rt, token_budget=16))
    got = [int(x) for x in srv.stream(prompts[1], SamplingParams(max_tokens=6)) if not isinstance(x, tuple)]
    srv.close()
    assert got == outs[1]
