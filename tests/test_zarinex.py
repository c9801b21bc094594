"""Zarinex without a GPU: configuration and registry, constants and layout of its layers, the oracle's sensitivity to the faults the
GPU tests look for, generation by the scheduler and the servers over the oracle."""
import json

import pytest
import torch
import zarinex_reference as zr
from gidisun_cases import OracleRuntime
from zarinex_cases import BEACON, FULL, again, beacon_tensors, clear_routes, config, forget, latent, moe, scan, tensors, tokens

from pocketllm_b200.models import mixer_layers as ml
from pocketllm_b200.models import registry
from pocketllm_b200.models import zarinex as zx
from pocketllm_b200.runtime.batching import BatchEngine
from pocketllm_b200.server.engine import SamplingParams, ServingEngine

_S, _L = scan(moe(experts=3)), latent(moe(experts=4))
SMALL = config([_S, _L, forget(), again(_S, 0), again(_L, 1)], width=40)


def test_config_registry_and_checkpoint_folder(tmp_path):
    c = zx.ZarinexConfig.from_dict(FULL)
    assert c.alpha == 2.3 and [c.owner(i) for i in range(9)] == [0, 1, 0, 3, 4, 3, 1, 7, 0]
    assert c.layers[3].shared_ff == 0 and c.layers[1].shared_ff == 130 and c.layers[4].mlp is None
    t = tensors(FULL)
    assert set(t) == set(zx.tensor_plan(c)) and not any(n.startswith(("l2.", "l5.", "l6.", "l8.")) for n in t)
    assert t["l7.mix.x"].shape == (40 + 2 * 21, 33) and t["l1.mix.g"].shape == (3 * 26, 88) and t["l3.mix.lower"].shape == (100,)
    assert "l4.norm2" not in t and "l4.rg2" not in t and "l3.mlp.shared.up" not in t and "head" not in t and t["l0.rg2"].shape == (88, 88)
    zx.save_checkpoint(tmp_path, c, t)
    assert json.loads((tmp_path / "config.json").read_text()) == FULL
    assert zx.ZarinexConfig.load(tmp_path) == c
    assert registry.folder_architecture(tmp_path) == "Zarinex" and "Zarinex" in registry.architectures()
    back = zx.load_tensors(tmp_path)
    assert all(torch.equal(back[k], t[k]) for k in t)
    from pocketllm_b200.server import openai as oa
    assert oa.detect_model_kind(str(tmp_path)) == "mixer"


@pytest.mark.parametrize("bad", [
    dict(layers=[]),
    dict(layers=[{"type": "mamba2", "mixer": {}, "mlp": None}]),
    dict(layers=[{"type": "hgrn2", "mixer": {"heads": 1, "dim": 8}, "mlp": None}]),
    dict(layers=[scan(conv=0)]), dict(layers=[latent(q_rank=0)]), dict(layers=[forget(vdim=0)]),
    dict(layers=[scan(moe(experts=3, top=4))]), dict(layers=[scan(moe(experts=0))]), dict(layers=[scan({"kind": "dense", "ff": 8})]),
    dict(layers=[scan(), again(scan(inner=61), 0)]), dict(layers=[scan(), again(forget(), 0)]), dict(layers=[scan(), again(scan(moe()), 0)]),
    dict(layers=[again(scan(), 0)]), dict(layers=[again(scan(), 1), again(scan(), 0)]), dict(layers=[scan(), again(scan(), 2)]),
    dict(architecture="Zemozen"),
])
def test_config_refuses_what_it_does_not_know(bad):
    with pytest.raises(ValueError):
        zx.ZarinexConfig.from_dict(FULL | bad)


def test_missing_and_misshapen_tensors_are_refused():
    c, t = zx.ZarinexConfig.from_dict(FULL), tensors(FULL)
    with pytest.raises(KeyError, match="l0.mix.dt.b"):
        zx.build_model(c, {k: v for k, v in t.items() if k != "l0.mix.dt.b"}, device="cpu")
    with pytest.raises(ValueError, match="l1.mlp.shared.gate"):
        zx.build_model(c, t | {"l1.mlp.shared.gate": t["l1.mlp.shared.gate"][:-1]}, device="cpu")


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_layers_of_the_model(dtype):
    """Constants, columns and memory of the layers."""
    c, t = zx.ZarinexConfig.from_dict(FULL), tensors(FULL)
    m = zx.build_model(c, t, device="cpu", slots=3, pages=5, dtype=dtype)
    assert m.post.alpha == 2.3 and m.windows() == {0} and m.post.freq.tolist() == pytest.approx([10000.0 ** (-2 * i / 88) for i in range(44)])
    assert torch.equal(m.head.w[:101, :88].float(), t["embed"].float())
    own = lambda L: L.mixer.S if hasattr(L.mixer, "S") else L.mixer.cache
    for i, j in ((2, 0), (8, 0), (5, 3), (6, 1)):      # the same weights, memory of its own
        a, b = m.layers[i], m.layers[j]
        assert a.mixer.proj is b.mixer.proj and a.mlp is b.mlp and a.norm1 is b.norm1 and a.shift is b.shift and a.gate_b is b.gate_b
        assert own(a) is not own(b) and own(a).shape == own(b).shape and a.before is not b.before
    s = m.layers[2].mixer
    assert s.S.shape == (3, 60, 10) and s.ring.shape == (3, 3, 60) and s.desc["S"] == s.S.data_ptr() and s.desc["ring"] == s.ring.data_ptr()
    p = m.layers[0].mixer
    assert p.desc["S"] != s.desc["S"] and (p.proj.at, p.proj.split) == ({"gate": 0, "x": 88, "z": 148}, 88)
    scale = 1.4426950408889634 if dtype == torch.bfloat16 else 1.0
    assert torch.allclose(p.const["A"], -torch.exp(t["l0.mix.A_log"].float()) * scale, rtol=1e-6)
    w = t["l0.mix.dt"].to(dtype)
    assert torch.equal(p.dt.w[:60, :7], w) and (p.dt.w[:60, 7:32] == 0).all() and p.dt.K == (64 if dtype == torch.bfloat16 else 32)
    assert dtype == torch.float32 or torch.equal(p.dt.w[:60, 32:39], w)
    a = m.layers[1].mixer
    assert (a.q_rank, a.R, a.window, a.gated) == (30, 0, 0, True) and a.proj.at == {"gate": 0, "dq": 88, "dkv": 120, "g": 164} and a.cache.shape == (5, 64, 64)
    assert a.uq.N == 3 * 64 and torch.equal(a.uq.w.view(3, 64, 64)[1, :22, :30], t["l1.mix.uq"].to(dtype)[22:44]) and (a.uq.w.view(3, 64, 64)[:, 22:] == 0).all()
    h = m.layers[3].mixer
    assert h.desc["qscale"] == 1.0 and (h.desc["oq"], h.desc["of"], h.desc["ov"]) == (88, 188, 288) and h.S.shape == (3, 5, 20, 28)
    e = m.layers[1].mlp
    assert e.route == ml.mo.Router(4, 3, score="softmax", renorm=True, on_output=True) and e.shared.ff == 256 and m.layers[3].mlp.shared is None
    assert e.router.at == {"router": 0, "gate": 4} and torch.equal(e.bias, t["l1.mlp.router.b"].float()) and m.layers[4].mlp is None
    assert m.layers[4].gate_b[1] is None and torch.equal(m.layers[4].gate_b[0], t["l4.rg1.b"].float()) and m.layers[7].before.shape == (3, 88)


def test_two_inputs_of_one_product():
    a, b, c = torch.randn(5, 9), torch.randn(3, 9), torch.randn(4, 9)
    f = ml.FusedLinear([("b", b), ("c", c)], torch.float32, "cpu", align=4, beside=[("a", a)])
    assert f.at == {"a": 0, "b": 8, "c": 12} and (f.split, f.N, f.K) == (8, 16, 64)
    assert torch.equal(f.w[:5, :9], a) and torch.equal(f.w[8:11, :9], b) and torch.equal(f.w[12:, :9], c) and (f.w[:, 9:] == 0).all()
    with pytest.raises(ValueError):
        ml.FusedLinear([("b", b)], torch.float32, "cpu", beside=[("a", a[:, 1:])])


@pytest.mark.parametrize("fault", ["position", "shift", "gated", "shared_state", "q_norm", "out_gate", "skip", "lower", "router_bias", "shared"])
def test_oracle_notices_faults(fault):
    """The tests' weights make each of these faults visible."""
    t = tensors(SMALL, gain=3.0)
    if fault == "router_bias":
        t = clear_routes(SMALL, t)
    seq = tokens(14, SMALL["vocab"], 3)
    good = zr.PlainModel(SMALL, t).logits(seq)
    zr.MUTATE.add(fault)
    try:
        bad = zr.PlainModel(SMALL, t).logits(seq)
    finally:
        zr.MUTATE.clear()
    d = (good - bad).pow(2).mean(-1).sqrt() / good.std()
    assert d.max() > 0.1


def test_oracle_sees_one_key_out_of_hundreds():
    cfg = config([latent()])
    t = beacon_tensors(cfg)
    seq = tokens(300, cfg["vocab"], 3, low=1)
    seq[20] = BEACON
    a, b = (zr.PlainModel(cfg, t).logits(s) for s in (seq, seq[:20] + [5] + seq[21:]))
    d = (a - b).pow(2).mean(-1).sqrt() / a.std()
    assert d[:20].max() == 0 and d[22:].min() > 0.1


def test_routes_of_the_test_weights_are_clear():
    t = clear_routes(FULL, tensors(FULL))
    m = zr.PlainModel(FULL, t)
    gaps, seen, turned = [], set(), 0
    plain = zr.route

    def watch(w, cfg, h):
        nonlocal turned
        raw = w["router"] @ h
        z, k = raw + w["router.b"], cfg["router"]["top"]
        s = z.sort(descending=True).values
        if k < len(s):
            gaps.append(float(s[k - 1] - s[k]))
        out = plain(w, cfg, h)
        seen.update((len(z), e) for e, _ in out)
        turned += {e for e, _ in out} != set(torch.topk(raw, k).indices.tolist())
        return out
    zr.route = watch
    try:
        m.logits(tokens(25, FULL["vocab"], 1))
    finally:
        zr.route = plain
    assert min(gaps) > 0.05 and turned > 10 and {(5, 4), (4, 3)} <= seen


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
