"""Gidisun without a GPU: configuration and registry, the oracle's sensitivity to the faults the GPU tests look for, page and
slot bookkeeping, work lists of mixed batches, the batching scheduler and the servers over the oracle."""
import json
import threading

import mixer_reference as mr
import numpy as np
import pytest
import torch
from gidisun_cases import BEACON, OracleRuntime, beacon_tensors, config, gla, latent, mlstm, tensors, tokens

from pocketllm_b200.models import gidisun as gd
from pocketllm_b200.models import registry
from pocketllm_b200.models.mixer_layers import rotary_frequencies
from pocketllm_b200.runtime.batching import BatchEngine
from pocketllm_b200.runtime.mixer_runtime import plan_portions
from pocketllm_b200.runtime.pd_scheduler import PDScheduler
from pocketllm_b200.runtime.request_cache import CacheFull, RequestCache
from pocketllm_b200.server.engine import SamplingParams, ServingEngine

CFG = config([mlstm(), latent(ff=100), gla()])


def test_config_registry_and_checkpoint_folder(tmp_path):
    c = gd.GidisunConfig.from_dict(CFG)
    assert c.to_dict()["layers"][1]["mlp"]["ff"] == 100 and c.layers[0].mlp is None
    t = tensors(CFG)
    assert set(t) == set(gd.tensor_plan(c))
    gd.save_checkpoint(tmp_path, c, t)
    assert gd.GidisunConfig.load(tmp_path) == c
    assert registry.folder_architecture(tmp_path) == "Gidisun" and "Gidisun" in registry.architectures()
    back = gd.load_tensors(tmp_path)
    assert all(torch.equal(back[k], t[k]) for k in t)
    from pocketllm_b200.server import openai as oa
    assert oa.detect_model_kind(str(tmp_path)) == "mixer"
    other = tmp_path / "other"
    other.mkdir()
    (other / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    assert registry.folder_architecture(other) is None
    with pytest.raises(KeyError):
        registry.build_runtime(other)


@pytest.mark.parametrize("bad", [
    dict(layers=[{"type": "conv", "mixer": {}, "mlp": None}]),
    dict(layers=[{"type": "gla", "mixer": {"heads": 1, "dim": 8, "vdim": 8}, "mlp": None}]),
    dict(layers=[mlstm() | {"mlp": {"kind": "routed", "ff": 8}}]),
    dict(layers=[latent(rot=10) | {"mixer": latent(rot=10)["mixer"] | {"rot_dim": 8}}]),
])
def test_config_refuses_what_it_does_not_know(bad):
    with pytest.raises(ValueError):
        gd.GidisunConfig.from_dict(CFG | bad)


def test_missing_and_misshapen_tensors_are_refused():
    c, t = gd.GidisunConfig.from_dict(CFG), tensors(CFG)
    with pytest.raises(KeyError, match="l1.mix.sink"):
        gd.build_model(c, {k: v for k, v in t.items() if k != "l1.mix.sink"}, device="cpu")
    with pytest.raises(ValueError, match="l0.mix.q"):
        gd.build_model(c, t | {"l0.mix.q": t["l0.mix.q"][:-1]}, device="cpu")


@pytest.mark.parametrize("dims,base,scaling", [
    (12, 5000.0, {"factor": 3.0, "original": 300, "fast": 20.0, "slow": 1.5}),
    (64, 1e6, {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
    (8, 100.0, {"factor": 1.0, "original": 64, "fast": 4.0, "slow": 1.0}),
    (2, 30.0, {"factor": 2.5, "original": 64, "fast": 2.0, "slow": 1.0}),
    (16, 10000.0, None),
])
def test_rotary_frequencies(dims, base, scaling):
    f, mag = rotary_frequencies(dims, base, scaling)
    want, wm = mr.yarn_frequencies({"dims": dims, "base": base, "scaling": scaling})
    assert torch.allclose(f, want, rtol=1e-12) and mag == pytest.approx(wm, rel=1e-12)


def test_oracle_notices_window_and_sink_faults():
    """The beacon weights make a window that is one token off, and a sink left out, visible (the GPU tests rely on it)."""
    cfg = config([latent(window=29)])
    t = beacon_tensors(cfg)
    seq = tokens(80, cfg["vocab"], 3, low=1)
    seq[20] = BEACON
    good = mr.PlainModel(cfg, t).logits(seq)
    for fault, where in (("window", 20 + 29), ("sink", 10)):
        mr.MUTATE.add(fault)
        try:
            bad = mr.PlainModel(cfg, t).logits(seq)
        finally:
            mr.MUTATE.clear()
        rel = (good - bad).pow(2).mean(-1).sqrt() / good.std()
        assert rel[where] > (0.3 if fault == "window" else 0.05), (fault, float(rel[where]))
    inside = mr.PlainModel(cfg, t).logits(seq[:20] + [5] + seq[21:])
    d = (good - inside).pow(2).mean(-1).sqrt() / good.std()
    assert d[48] > 0.3 and d[49] < 1e-9                     # position 20 is seen up to position 48


# ---- pages and slots ----

def test_request_cache_hands_out_and_takes_back():
    c = RequestCache(2, 5, page=4, device=None)
    c.reserve({"a": 5, "b": 1})
    assert c.free_pages == 2 and c.free_slots == 0
    assert c.table[c.slot("a"), 0] != c.table[c.slot("a"), 1]
    with pytest.raises(CacheFull):
        c.reserve({"c": 1})
    with pytest.raises(CacheFull):
        c.reserve({"a": 8, "b": 13})                        # needs three pages, two are free: nothing changes
    assert c.free_pages == 2
    c.reserve({"a": 8})
    assert c.free_pages == 2                                # fits into the pages it has
    c.advance("a", 8)
    old = set(c.table[c.slot("a"), :2].tolist())
    slot = c.slot("a")
    c.release("a")
    assert "a" not in c and c.free_pages == 4
    c.reserve({"d": 16})
    assert c.slot("d") == slot and old <= set(c.table[slot, :4].tolist()) and c.length["d"] == 0
    used = c.table[c.slot("d"), :4].tolist() + c.table[c.slot("b"), :1].tolist()
    assert len(set(used)) == 5                              # nobody shares a page


def test_plan_portions():
    p = plan_portions([1, 70, 8, 130], [9, 0, 100, 37], [2, 0, 1, 3], windows=[0, 40], rows_max=8, chunk=64, tile=128)
    assert p["T"] == 209 and p["pos"][0] == 9 and p["pos"][1] == 0 and p["pos"][-1] == 166
    assert p["short"] == [(0, 1, 2, 9), (71, 8, 1, 100)] and p["rows"] == [0] + list(range(71, 79))
    assert p["long"] == [(1, 70, 0, 0), (79, 130, 3, 37)] and p["chunk0"] == [0, 2]
    assert p["chunks"] == [(1, 64, 0, 0), (65, 6, 0, 1), (79, 64, 1, 0), (143, 64, 1, 1), (207, 2, 1, 2)]
    assert p["tiles"] == [(1, 70, 0, 0), (79, 128, 1, 0), (207, 2, 1, 0)]
    assert p["gather"][0] == [(0, 0), (70, 0)] and p["total"][0] == 70 + 167
    assert p["gather"][40] == [(0, 0), (70, 0)] and p["longest"][40] == 167
    assert plan_portions([10], [100], [0], windows=[40])["gather"][40] == [(0, 61)]
    assert np.flatnonzero(p["last"] >= 0).tolist() == [0, 70, 78, 208] and p["last"][78] == 1


# ---- scheduling ----

def test_next_batch_decodes_first_and_cuts_prompts():
    s = PDScheduler()
    left = {"a": 10, "b": 3, "c": 5}
    for r in "abc":
        s.submit(r)
    room = {"a", "b"}
    take = lambda: s.next_batch(4, 8, lambda r: left[r], lambda r: r in room)
    assert take() == [("a", "prefill", 8)]
    left["a"] = 2
    s.prefill_more("a")
    assert take() == [("a", "prefill", 2), ("b", "prefill", 3)]    # c has no room
    s.prefill_done("a")
    s.prefill_done("b")
    assert take() == [("a", "decode", 1), ("b", "decode", 1)]
    s.requeue_decode("a")
    s.finish("b")
    room.add("c")
    assert take() == [("a", "decode", 1), ("c", "prefill", 5)]
    s.drop("c")
    assert take() == [] and s.pending() == (0, 0)


def test_batch_engine_matches_plain_generation():
    t = tensors(CFG)
    rt = OracleRuntime(CFG, t, max_requests=3, pages=12, page=16)
    eng = BatchEngine(rt, token_budget=24, burst=4)
    prompts = [tokens(n, CFG["vocab"], n) for n in (5, 41, 1, 17, 30, 9)]
    outs = eng.run(prompts, [SamplingParams(max_tokens=m) for m in (7, 12, 20, 3, 6, 9)])
    m = mr.PlainModel(CFG, t)
    for p, o, n in zip(prompts, outs, (7, 12, 20, 3, 6, 9)):
        assert o == m.generate(p, n)
    assert rt.cache.free_pages == 12 and rt.cache.free_slots == 3
    assert eng.stats["mixed_steps"] > 0 and eng.stats["burst_steps"] > 0 and any(len(c) == 3 for c in rt.calls)
    assert all(sum(c) <= 24 for c in rt.calls)


def test_batch_engine_stop_tokens_sampling_and_limits():
    t = tensors(CFG)
    m = mr.PlainModel(CFG, t)
    p = tokens(6, CFG["vocab"], 1)
    ref = m.generate(p, 12)
    eng = BatchEngine(OracleRuntime(CFG, t, max_requests=2, pages=3, page=16), burst=8)
    assert eng.run([p], [SamplingParams(max_tokens=12, stop_token_ids=(ref[4],))]) == [ref[:ref.index(ref[4]) + 1]]
    a, b = eng.run([p, p], [SamplingParams(max_tokens=6, temperature=1.0, seed=3), SamplingParams(max_tokens=6, temperature=1.0, seed=3)])
    assert a == b
    (lp,) = eng.run([p], [SamplingParams(max_tokens=2, logprobs=2)])
    assert [x.token for x in lp] == ref[:2] and len(lp[0].top) == 2 and lp[0].top[0][0] == ref[0]
    assert len(eng.run([p], [SamplingParams(max_tokens=500)])[0]) == 48 - 6 + 1      # as long as the cache has room
    with pytest.raises(ValueError):
        eng.submit([1] * 49, SamplingParams())
    with pytest.raises(ValueError):
        eng.submit([], SamplingParams())
    with pytest.raises(ValueError):
        eng.submit([CFG["vocab"]], SamplingParams())
    rid = eng.submit(p, SamplingParams(max_tokens=9))
    eng.step()
    eng.cancel(rid)
    assert eng.idle and eng.rt.cache.free_pages == 3 and eng.rt.cache.free_slots == 2


def test_serving_engine_runs_requests_together_and_survives_a_failed_step():
    from pocketllm_b200.server.backends import MixerBackend
    t = tensors(CFG)
    rt = OracleRuntime(CFG, t, max_requests=3, pages=12, page=16)
    be = MixerBackend(rt, token_budget=16)
    srv = ServingEngine(be)
    m = mr.PlainModel(CFG, t)
    prompts = [tokens(n, CFG["vocab"], 50 + n) for n in (12, 3, 20, 7)]
    got: dict[int, list] = {}

    def ask(i):
        got[i] = [int(x) for x in srv.stream(prompts[i], SamplingParams(max_tokens=8)) if not isinstance(x, tuple)]
    th = [threading.Thread(target=ask, args=(i,)) for i in range(4)]
    [x.start() for x in th]
    [x.join(60) for x in th]
    for i, p in enumerate(prompts):
        assert got[i] == m.generate(p, 8)
    assert rt.cache.free_slots == 3
    rt.fail_next = True
    with pytest.raises(RuntimeError, match="scripted"):
        list(srv.stream(prompts[0], SamplingParams(max_tokens=4)))
    with pytest.raises(ValueError):
        list(srv.stream([], SamplingParams(max_tokens=4)))
    ask(1)
    assert got[1] == m.generate(prompts[1], 8)
    it = srv.stream(prompts[2], SamplingParams(max_tokens=40))
    next(it), next(it)
    it.close()                                             # the client went away
    srv.close()
    assert list(be.generate(prompts[1], SamplingParams(max_tokens=5))) == got[1][:5]
    assert rt.cache.free_slots == 3 and rt.cache.free_pages == 12


def test_kernel_set_is_compiled_only_when_needed(tmp_path, monkeypatch):
    from pocketllm_b200 import build
    calls = []
    monkeypatch.setattr(build, "OUT", tmp_path / "_C")
    monkeypatch.setattr(build, "OBJ", tmp_path / "build" / "obj")
    monkeypatch.setattr(build, "_compile_one", lambda s, h, e, v: calls.append(s) or s)
    monkeypatch.setattr(build, "_link", lambda objs, out, shared, extra, v: out.write_bytes(b"x"))
    lib = build.ensure_kernels("mixer")
    assert lib.name == "libpocket_kernels_mixer.so" and len(calls) == len(build.KERNEL_SETS["mixer"])
    assert build.ensure_kernels("mixer") == lib and len(calls) == len(build.KERNEL_SETS["mixer"])
    full = build.OUT / "libpocket_kernels.so"
    full.write_bytes(b"y")
    assert build.ensure_kernels("mixer") == lib            # no record of what the full library was built from
    build._write_stamp(full, [build.CSRC / s for s in build.KERNEL_SETS["mixer"]], build._headers_digest())
    assert build.ensure_kernels("mixer") == full


def test_argument_kinds_match_the_launchers():
    """The ctypes prototypes of `ops.mixer_ops` against the C signatures in the sources."""
    import re

    from pocketllm_b200 import build
    from pocketllm_b200.ops import mixer_ops as mo
    src = "\n".join((build.CSRC / s).read_text() for s in build.KERNEL_SETS["mixer"])
    for name, kinds in mo._SIGNATURES.items():
        m = re.search(r"PK_API int " + name + r"\(([^)]*)\)", src)
        params = [p.strip() for p in m.group(1).split(",")]
        assert params[-1] == "cudaStream_t stream"
        got = "".join("p" if "*" in p else "f" if p.startswith("float") else "i" for p in params[:-1])
        assert got == kinds, name
