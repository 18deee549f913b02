"""Dorevik through the engine on the CPU (PyTorch operators) against the plain statement in tests/dorevik_oracle.py:
configuration and loading, schedules, pages and state rows that are used again, generation."""
import copy
import math

import pytest
import torch

import dorevik_cases as S
import dorevik_oracle as O
from fllm_b200.config import EngineConfig, ModelConfig, MoeSpec, ParallelConfig, RopeScaling, preset, scaled_inv_freq
from fllm_b200.runtime.engine import LLMEngine
from fllm_b200.runtime.request import SamplingParams

TOL = 2e-5


@pytest.mark.parametrize("name", list(S.CONFIGS))
def test_prompt_and_decoding_match_the_oracle(name):
    cfg, w, toks, want = S.expected(name, 41, 1)
    rp = S.TraceReplay(S.engine(cfg, w))
    assert S.error(S.feed(rp, "a", toks, []), want) < TOL                                   # one portion
    assert S.error(S.feed(rp, "b", toks, range(1, 41)), want) < TOL                         # token by token
    assert S.error(S.feed(rp, "c", toks, [2, 4, 9, 15, 16, 17, 33]), want) < TOL            # portions around the 16-token pages
    assert len(rp.eng.blocks.free) == rp.eng.blocks.num_blocks


def test_bf16_serving_is_close():
    for name in ("odd", "tensor-cores"):
        cfg, w, toks, want = S.expected(name, 41, 1, True)
        assert S.error(S.feed(S.TraceReplay(S.engine(cfg, w, f32=False)), "a", toks, [7]), want) < 8e-2


def test_a_token_in_a_window_or_a_state_shows_in_the_logits():
    """The weights are sharp enough for the other tests to mean something: the last logits move far beyond the tolerances when a
    token inside the reach of the windows changes, and when the first token of a sequence of recurrent layers does."""
    cfg, w, toks, want = S.expected("tensor-cores", 41, 1)
    slow = S.config([S.parallel(S.heads(2, 1, 8, 8, 2, 4), [0.97, 0.99], 8, 8)], 61, 40)
    ws, ts = S.tensors(slow), S.prompt(slow, 41, 2)
    for cfg, w, toks, place in ((cfg, w, toks, 0), (cfg, w, toks, 20), (cfg, w, toks, 39), (slow, ws, ts, 0)):
        want, other = O.forward(cfg, w, toks, torch.float64), list(toks)
        other[place] = (other[place] + 11) % cfg["vocab"]
        assert S.error(O.forward(cfg, w, other, torch.float64)[-1:], want[-1:]) > 50 * TOL, place


CHANGES = {
    "window": lambda c: c["layers"][0]["mixer"]["mask"].update(size=18), "left_window": lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=8),
    "scale": lambda c: c["layers"][0]["mixer"].update(scale=0.1), "diff": lambda c: c["layers"][2]["mixer"].update(diff=0.7),
    "decay": lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.004, 0.8, 0.9995]), "base": lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(base=40.0),
    "rot_dims": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=20), "factor": lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=9.0),
    "original": lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(original=100), "fast": lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(fast=3.0),
    "slow": lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(slow=0.1), "no_scaling": lambda c: c["layers"][0]["mixer"]["rot"].pop("scaling"),
    "top": lambda c: c["layers"][0]["mlp"]["router"].update(top=2), "no_shared": lambda c: c["layers"][0]["mlp"].pop("shared"),
    "cap": lambda c: c.update(logit_softcap=3.0), "eps": lambda c: c["norm"].update(eps=0.3), "no_mlp": lambda c: c["layers"][1].update(mlp=None),
    "order": lambda c: c["layers"].insert(0, c["layers"].pop(2)),
}


@pytest.mark.parametrize("change", list(CHANGES))
def test_every_constant_is_read_from_the_configuration(change):
    """Another value of one constant: the engine follows the oracle, and the logits move."""
    base, w, toks, want = S.expected("odd", 41, 1)
    cfg = copy.deepcopy(base)
    CHANGES[change](cfg)
    if change == "order":
        w = S.tensors(cfg)
    moved = O.forward(cfg, w, toks, torch.float64)
    assert S.error(moved, want) > 50 * TOL
    assert S.error(S.feed(S.TraceReplay(S.engine(cfg, w)), "a", toks, [5, 20]), moved) < TOL


def test_mixed_batches_pages_and_rows_are_reused():
    """Four live requests of unequal progress in every step; finished ones give pages and state rows to later ones."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, blocks=12, max_len=96)
    rp = S.TraceReplay(eng)
    g = torch.Generator().manual_seed(5)
    reqs = {f"r{i}": S.prompt(cfg, n, 100 + i) for i, n in enumerate((37, 5, 50, 18, 33, 2, 47))}
    want = {k: O.forward(cfg, w, v, torch.float64) for k, v in reqs.items()}
    at, waiting, live = {k: 0 for k in reqs}, list(reqs), []
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-len(reqs[k]) // 16) for k in live + waiting[:1]) <= 12:
            live.append(waiting.pop(0))
        entries, ends = [], []
        for k in live:
            if len(live) > 1 and entries and int(torch.randint(0, 5, (1,), generator=g)) == 0:
                continue                                                                     # left out of this step
            n = min(int(torch.randint(1, 14, (1,), generator=g)), len(reqs[k]) - at[k]) if at[k] % 2 else 1
            entries.append(dict(id=k, tokens=reqs[k][at[k]:at[k] + n], want=list(range(n))))
            if at[k] + n == len(reqs[k]):
                ends.append(k)
        lg, row = rp.step(entries, ends), 0
        for e in entries:
            n, k = len(e["tokens"]), e["id"]
            assert S.error(lg[row:row + n], want[k][at[k]:at[k] + n]) < TOL, (k, at[k])
            at[k] += n
            row += n
        live = [k for k in live if k not in ends]
    assert len(eng.blocks.free) == 12 and len(eng.blocks.state_free) == 4


def test_generation_through_the_scheduler_gives_back_pages_behind_the_windows():
    """Greedy text of unequal requests with chunked prompts in a pool that is too small for whole sequences: each token is the
    oracle's best one, and the pages no window reaches any more are used again."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, chunk=16, seqs=2, spare=4, blocks=10)
    assert eng.scheduler.window == 33
    prompts = [S.prompt(cfg, n, n) for n in (3, 75, 17, 60)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=30, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = O.forward(cfg, w, p + o, torch.float64)[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert len(o) == 30 and float(gap.max()) < 1e-4 * float(lg.std())


def test_checkpoint_directory_and_config(tmp_path):
    cfg, w, toks, want = S.expected("odd", 41, 1)
    mc, weights, tok = S.load_model(S.write_checkpoint(tmp_path / "m", cfg, w), "cpu", dtype=torch.float32)
    assert tok is None and mc.arch == "dorevik" and mc.native_f32 and mc.native_part == "maps" and mc.has_recurrent and mc.has_row_cache
    assert [mc.layer_kind(i) for i in range(4)] == ["maps", "maps+lightning"] * 2 and [mc.ffn_kind(i) for i in range(4)] == ["moe", "glu", "none", "moe"]
    assert ModelConfig.from_dict(mc.to_dict()) == mc
    assert mc.moe_of(0) == MoeSpec(7, 3, "deepseek_v3", act="swiglu", weigh_input=True, fp32_router=True) and weights.layers[3].moe.top == 1
    from fllm_b200.models.recurrent import RecurrentState
    from fllm_b200.models.row_cache import RowCache, RowSpec
    specs = RowCache.specs(mc, range(4))
    assert specs == [RowSpec(64, 4, 64, 2), RowSpec(64, 5, 64, 5), RowSpec(64, 2, 64, 1), RowSpec(64, 2, 64, 2)]
    assert RowCache.bytes_per_block(specs, 16) == 16 * 2 * 64 * (6 + 10 + 3 + 4)
    assert RecurrentState.bytes_per_slot(mc, range(4)) == 4 * (3 * 13 * 10 + 24 * 40)
    assert RecurrentState(mc, range(4), 3, "cpu").nbytes() == 3 * RecurrentState.bytes_per_slot(mc, range(4))
    assert weights.nbytes() > sum(t.numel() for t in w.values()) * 4
    bad = dict(w)
    bad["l1.mix.right.v"] = bad["l1.mix.right.v"][:-1]
    with pytest.raises(ValueError):
        S.load_tensors(cfg, bad, "cpu", torch.float32)
    breaks = [lambda c: c["layers"][0]["mixer"].update(kv_heads=4), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), lambda c: c["layers"][1].update(type="other"),
              lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
              lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]), lambda c: c["layers"][0]["mlp"]["router"].update(top=8),
              lambda c: c["layers"][1]["mlp"].update(kind="other")]
    for change in breaks:
        broken = copy.deepcopy(cfg)
        change(broken)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(broken)


def test_residual_after_every_layer():
    """The engine's residual of a model cut behind each of its layers."""
    cfg, w, toks, _ = S.expected("tensor-cores", 41, 1)
    want = []
    O.forward(cfg, w, toks, torch.float64, want)
    for n in range(1, len(cfg["layers"]) + 1):
        cut = dict(cfg, layers=cfg["layers"][:n])
        eng = S.engine(cut, dict(w, **{"final.norm": torch.ones(cfg["width"]), "head": torch.eye(cfg["vocab"], cfg["width"])}))
        eng.decoder.capture_hidden = True
        S.feed(S.TraceReplay(eng), "a", toks, [])
        got = eng.decoder.last_hidden.double()[:, :cfg["width"]]
        assert float((got - O.rms(want[n - 1], cfg["norm"]["eps"])).abs().max()) < 1e-4, n


def test_scaled_rotation_frequencies():
    rot = dict(base=500.0, dims=24, scaling=dict(factor=3.0, original=40, fast=8.0, slow=0.5))
    f, factor = O.frequencies(rot)
    got, got_factor = scaled_inv_freq(24, 500.0, RopeScaling("yarn", 3.0, original_max_position=40, beta_fast=8.0, beta_slow=0.5))
    assert torch.allclose(torch.tensor(got), torch.tensor(f), rtol=1e-12) and abs(factor - got_factor) < 1e-12 and factor == 0.1 * math.log(3.0) + 1
    assert f[0] == 1.0 and abs(f[-1] * 3 - 500.0 ** (-22 / 24)) < 1e-12 and f[0] / got[3] > 1


def test_preset_runs_with_random_weights():
    eng = LLMEngine(preset("dorevik-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64, max_num_seqs=2), device="cpu")
    out = eng.generate([[1, 2, 3], [4, 5]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert [len(o) for o in out] == [5, 5]
    eng = LLMEngine(preset("dorevik-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64, max_num_seqs=2), device="cpu")
    assert out == eng.generate([[1, 2, 3], [4, 5]], SamplingParams(max_tokens=5, ignore_eos=True))


def test_tensor_parallel_ranks_are_refused():
    with pytest.raises(NotImplementedError):
        LLMEngine(preset("dorevik-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64), ParallelConfig(tp=2), device="cpu")
