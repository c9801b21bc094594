"""Pezarax without a GPU: configuration and registry, the order of repeated layers, the oracle's sensitivity to the faults the
GPU tests look for, generation by the scheduler and the servers over the oracle."""
import json

import pezarax_reference as pr
import pytest
import torch
from gidisun_cases import OracleRuntime
from pezarax_cases import BEACON, FULL, attention, beacon_tensors, clear_routes, config, moe, retention, tensors, tokens

from pocketllm_b200.models import pezarax as pz
from pocketllm_b200.models import registry
from pocketllm_b200.runtime.batching import BatchEngine
from pocketllm_b200.server.engine import SamplingParams, ServingEngine

SMALL = config([retention(mlp=moe(experts=3, top=1)), attention(chunk=7)], width=40, loop=(0, 2, 2))


def test_config_registry_and_checkpoint_folder(tmp_path):
    c = pz.PezaraxConfig.from_dict(FULL)
    assert c.loop == (1, 3, 3) and c.layers[3].top == 1 and c.layers[2].mlp is None
    t = tensors(FULL)
    assert set(t) == set(pz.tensor_plan(c)) and t["l1.mlp.e4.down"].shape == (88, 36)
    pz.save_checkpoint(tmp_path, c, t)
    assert json.loads((tmp_path / "config.json").read_text()) == FULL
    assert pz.PezaraxConfig.load(tmp_path) == c
    assert registry.folder_architecture(tmp_path) == "Pezarax" and "Pezarax" in registry.architectures()
    back = pz.load_tensors(tmp_path)
    assert all(torch.equal(back[k], t[k]) for k in t)
    from pocketllm_b200.server import openai as oa
    assert oa.detect_model_kind(str(tmp_path)) == "mixer"


@pytest.mark.parametrize("bad", [
    dict(layers=[{"type": "mlstm", "mixer": {}, "mlp": None}]),
    dict(layers=[{"type": "retention", "mixer": {"heads": 1, "dim": 8, "vdim": 8}, "mlp": None}]),
    dict(layers=[retention(heads=2) | {"mixer": retention(heads=3)["mixer"] | {"heads": 2}}]),
    dict(layers=[retention(rot=5)]),
    dict(layers=[attention(dim=8, rot=10)]),
    dict(layers=[attention(heads=3, kv=2)]),
    dict(layers=[retention(mlp=moe(experts=3, top=4))]),
    dict(layers=[retention(mlp={"kind": "dense", "ff": 8})]),
    dict(loop={"start": 1, "stop": 5, "times": 2}),
    dict(loop={"start": 0, "stop": 1, "times": 0}),
    dict(architecture="Gidisun"),
])
def test_config_refuses_what_it_does_not_know(bad):
    with pytest.raises(ValueError):
        pz.PezaraxConfig.from_dict(FULL | bad)


def test_missing_and_misshapen_tensors_are_refused():
    c, t = pz.PezaraxConfig.from_dict(FULL), tensors(FULL)
    with pytest.raises(KeyError, match="l1.mix.lk2"):
        pz.build_model(c, {k: v for k, v in t.items() if k != "l1.mix.lk2"}, device="cpu")
    with pytest.raises(ValueError, match="l0.mlp.e3.up"):
        pz.build_model(c, t | {"l0.mlp.e3.up": t["l0.mlp.e3.up"][:-1]}, device="cpu")


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (0, 2, 3), (1, 3, 2), (3, 4, 2), (0, 4, 2)])
def test_runs_of_layers(loop):
    """Passes share weights, not states; the embedding output comes back once per further pass."""
    cfg = config(FULL["layers"], vocab=101, width=88, loop=loop)
    c = pz.PezaraxConfig.from_dict(cfg)
    want = pr.layer_runs(cfg)
    assert [i for i, _ in c.passes()] == [i for i, _ in want]
    m = pz.build_model(c, tensors(cfg), device="cpu", slots=2, pages=3)
    assert [L.reinject for L in m.layers] == [again for _, again in want]
    for j, (i, _) in enumerate(want):
        first = next(k for k, (x, _) in enumerate(want) if x == i)
        a, b = m.layers[first].mixer, m.layers[j].mixer
        assert a.proj is b.proj and m.layers[first].mlp is m.layers[j].mlp
    memory = [(L.mixer.S if hasattr(L.mixer, "S") else L.mixer.cache).data_ptr() for L in m.layers]
    assert len(set(memory)) == len(memory)


def test_attention_constants():
    """lambda from the four vectors, padding of keys and values in the cache, chunk and window from the mask."""
    from pocketllm_b200.models import mixer_layers as ml
    t, L = tensors(FULL), FULL["layers"][1]
    w = {n[len("l1.mix."):]: v for n, v in t.items() if n.startswith("l1.mix.")}
    m = ml.GroupedAttentionMixer(w, L["mixer"], 1e-5, torch.float32, "cpu", 4, 256, mask="chunk")
    assert m.desc["lambda_"] == pytest.approx(float(pr.diff_lambda({k: v.double() for k, v in w.items()}, 0.3)), rel=1e-12)
    assert m.desc["post"] == pytest.approx(0.7) and (m.desc["chunk"], m.desc["window"], m.nsplit) == (29, 0, 1)
    assert m.row == 2 * (2 * 24 + 32) and m.cache.shape == (4, 64, m.row)
    plain = {k: v for k, v in L["mixer"].items() if k != "diff"}
    half = {"q": w["q"][:6 * 22], "k": w["k"][:2 * 22], "v": w["v"], "o": w["o"]}
    m = ml.GroupedAttentionMixer(half, plain, 1e-5, torch.bfloat16, "cpu", 40, 2560)
    assert m.maps == 1 and (m.desc["chunk"], m.desc["window"]) == (0, 29) and "head_norm" not in m.desc


@pytest.mark.parametrize("fault,where", [("chunk", 29), ("lambda", 40), ("reinject", 3), ("weight", 3)])
def test_oracle_notices_faults(fault, where):
    """The tests' weights make a chunk that is one position off, a second map left out, a missing embedding and a weight at the
    wrong end of an expert visible."""
    if fault in ("reinject", "weight"):
        cfg = SMALL
        t = clear_routes(cfg, tensors(cfg))
        seq = tokens(10, cfg["vocab"], 3)
    else:
        cfg = config([attention(chunk=29)])
        t = beacon_tensors(cfg, chosen_map=1 if fault == "lambda" else 0)
        seq = tokens(60, cfg["vocab"], 3, low=1)
        seq[20 if fault == "chunk" else 35] = BEACON
    good = pr.PlainModel(cfg, t).logits(seq)
    pr.MUTATE.add(fault)
    try:
        bad = pr.PlainModel(cfg, t).logits(seq)
    finally:
        pr.MUTATE.clear()
    assert ((good - bad).pow(2).mean(-1).sqrt() / good.std())[where] > (0.05 if fault == "weight" else 0.1)


def test_oracle_sees_keys_to_the_end_of_their_chunk():
    cfg = config([attention(chunk=29)])
    for chosen in (0, 1):
        t = beacon_tensors(cfg, chosen_map=chosen)
        seq = tokens(60, cfg["vocab"], 3, low=1)
        seq[20] = BEACON
        a, b = (pr.PlainModel(cfg, t).logits(s) for s in (seq, seq[:20] + [5] + seq[21:]))
        d = (a - b).pow(2).mean(-1).sqrt() / a.std()
        assert d[28] > 0.1 and d[29] < 1e-9


def test_routes_of_the_test_weights_are_clear():
    t = clear_routes(FULL, tensors(FULL))
    m = pr.PlainModel(FULL, t)
    gaps, seen = [], set()
    plain = pr.route

    def watch(w, cfg, h):
        s = torch.sigmoid(w["router"] @ h).sort(descending=True).values
        gaps.append(float(s[cfg["router"]["top"] - 1] - s[cfg["router"]["top"]]))
        out = plain(w, cfg, h)
        seen.update(e for e, _ in out)
        return out
    pr.route = watch
    try:
        m.logits(tokens(25, FULL["vocab"], 1))
    finally:
        pr.route = plain
    assert min(gaps) > 0.02 and seen == set(range(5))


def test_generation_by_the_scheduler_and_the_server():
    from pocketllm_b200.server.backends import MixerBackend
    t = tensors(SMALL)
    rt = OracleRuntime(SMALL, t, max_requests=3, pages=12, page=16, plain=pr.PlainModel)
    m = pr.PlainModel(SMALL, t)
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


def test_descriptor_mirrors_the_header():
    """Field order and kinds of the ctypes descriptors against the C structs."""
    import ctypes
    import re

    from pocketllm_b200 import build
    from pocketllm_b200.ops import mixer_ops as mo
    for cls, file, name in ((mo.PagedAttention, "common/pk_paged.h", "PkPagedAttention"), (mo.StateMixer, "common/pk_state.cuh", "PkStateMixer")):
        body = re.search(r"struct " + name + r" \{(.*?)\};", (build.CSRC / file).read_text(), re.S).group(1)
        body = re.sub(r"//[^\n]*", "", body)
        want = []
        for decl in filter(None, (d.strip() for d in body.split(";"))):
            kind = ctypes.c_void_p if "*" in decl else ctypes.c_float if decl.startswith("float") else ctypes.c_int
            want += [(n.strip().split(" ")[-1].lstrip("*"), kind) for n in decl.split(",")]
        assert [(n.rstrip("_"), k) for n, k in cls._fields_] == want
