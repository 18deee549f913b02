"""Sovanex through the engine on the CPU (PyTorch operators) against the plain statement in tests/sovanex_oracle.py:
configuration and loading, schedules, pages and state rows that are used again, generation."""
import copy

import pytest
import torch

import sovanex_cases as S
import sovanex_oracle as O
from fllm_b200.config import ModelConfig, preset
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
    cfg, w, toks, want = S.expected("odd", 41, 1)
    assert S.error(S.feed(S.TraceReplay(S.engine(cfg, w, f32=False)), "a", toks, [7]), want) < 6e-2


def test_a_far_token_shows_in_the_logits():
    """The weights are sharp enough for the other tests to mean something: the oracle's last logits move far beyond the
    tolerances when one early token changes, with attention only (a lost key) and with recurrent layers only (a lost state)."""
    for name in ("attention-only", "delta-only", "odd"):
        cfg, w, toks, want = S.expected(name, 41, 1)
        for place in (0, 7, 16):
            other = list(toks)
            other[place] = (other[place] + 11) % cfg["vocab"]
            assert S.error(O.forward(cfg, w, other, torch.float64)[-1:], want[-1:]) > 50 * TOL, (name, place)


def test_mixed_batches_pages_and_rows_are_reused():
    """Four live requests of unequal progress in every step; finished ones give pages and state rows to later ones."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, blocks=12, max_len=96)
    rp = S.TraceReplay(eng)
    g = torch.Generator().manual_seed(5)
    reqs = {f"r{i}": S.prompt(cfg, n, 100 + i) for i, n in enumerate((37, 5, 50, 18, 33, 2, 47))}
    want = {k: O.forward(cfg, w, v, torch.float64) for k, v in reqs.items()}
    at, waiting, live, used = {k: 0 for k in reqs}, list(reqs), [], set()
    while waiting or live:
        held = lambda ks: sum(-(-len(reqs[k]) // 16) for k in ks)
        while waiting and len(live) < 4 and held(live + waiting[:1]) <= 12:
            live.append(waiting.pop(0))
        entries, ends = [], []
        for k in live:
            if len(live) > 1 and int(torch.randint(0, 5, (1,), generator=g)) == 0 and entries:
                continue                                                                     # left out of this step
            n = min(int(torch.randint(1, 14, (1,), generator=g)), len(reqs[k]) - at[k]) if at[k] % 2 else min(1, len(reqs[k]) - at[k])
            entries.append(dict(id=k, tokens=reqs[k][at[k]:at[k] + n], want=list(range(n))[::-1]))
            if at[k] + n == len(reqs[k]):
                ends.append(k)
        lg, row = rp.step(entries, ends), 0
        for e in entries:
            n = len(e["tokens"])
            assert S.error(lg[row:row + n].flip(0), want[e["id"]][at[e["id"]]:at[e["id"]] + n]) < TOL
            at[e["id"]] += n
            row += n
        used.update(eng.blocks.seqs[rp.live[k].seq_id].state_slot for k in live if k in rp.live)
        live = [k for k in live if k not in ends]
    assert used == {0, 1, 2, 3} and len(eng.blocks.state_free) == 4 and len(eng.blocks.free) == 12


def test_replay_refuses_what_does_not_fit():
    cfg, w, toks, _ = S.expected("odd", 41, 1)
    rp = S.TraceReplay(S.engine(cfg, w, blocks=2, max_len=64))
    with pytest.raises(RuntimeError):
        rp.step([dict(id="a", tokens=toks, want=[])])
    with pytest.raises(ValueError):
        rp.step([dict(id="b", tokens=[cfg["vocab"]], want=[])])
    with pytest.raises(ValueError):
        rp.step([dict(id="c", tokens=[1, 2], want=[2])])


def test_generation_follows_the_oracle():
    """Greedy generation through the scheduler: chunked prompts beside decoding requests, fewer state rows than requests."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, chunk=16, seqs=3, spare=8, blocks=40)
    prompts = [S.prompt(cfg, n, n) for n in (3, 29, 17, 8)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=9, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = O.forward(cfg, w, p + o, torch.float64)
        for j, t in enumerate(o):
            row = lg[len(p) - 1 + j]
            assert row.max() - row[t] <= 1e-4 * (row.max() - row.min())


def test_sampling_is_reproducible():
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    sp = SamplingParams(max_tokens=6, temperature=0.8, top_p=0.9, seed=3, ignore_eos=True)
    a = S.engine(cfg, w, spare=8).generate([S.prompt(cfg, 9, 1)], sp)
    assert a == S.engine(cfg, w, spare=8, chunk=4).generate([S.prompt(cfg, 9, 1)], sp) and len(a[0]) == 6


def test_checkpoint_directory_and_config(tmp_path):
    cfg, w, toks, want = S.expected("odd", 41, 1)
    mc, weights, tok = S.load_model(S.write_checkpoint(tmp_path / "m", cfg, w), "cpu", dtype=torch.float32)
    assert tok is None and mc.arch == "sovanex" and mc.native_f32 and mc.residual_streams == 3
    assert [mc.kv_source(i) for i in range(5)] == [0, 1, 0, 3, 0] and [mc.has_kv(i) for i in range(5)] == [True, False, False, False, False]
    assert [mc.ffn_kind(i) for i in range(5)] == ["glu", "glu", "none", "none", "glu"]
    assert ModelConfig.from_dict(mc.to_dict()) == mc
    from fllm_b200.models.row_cache import RowCache, RowSpec
    assert RowCache.specs(mc, range(5)) == [RowSpec(48)]                                             # 37 + 6, padded; shared by three layers
    bad = dict(w)
    bad["l1.mix.k"] = bad["l1.mix.k"][:-1]
    with pytest.raises(ValueError):
        S.load_tensors(cfg, bad, "cpu", torch.float32)
    with pytest.raises(KeyError):
        S.load_tensors(cfg, {k: v for k, v in w.items() if k != "l4.hc2.mix"}, "cpu", torch.float32)


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][2]["mixer"].update(kv_from=1), lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][4]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_rank=36),
    lambda c: c["layers"][2]["mixer"]["rot"].update(base=3.0), lambda c: c["layers"][1]["mixer"].update(heads=3),
    lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other")])
def test_configs_that_make_no_sense_are_refused(edit):
    cfg = copy.deepcopy(S.CONFIGS["odd"])
    edit(cfg)
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(cfg)


def test_preset_runs():
    from fllm_b200.config import EngineConfig
    from fllm_b200.runtime.engine import LLMEngine
    eng = LLMEngine(preset("sovanex-tiny"), EngineConfig(max_num_seqs=2, max_model_len=64, num_kv_blocks=16, max_num_batched_tokens=32), device="cpu")
    assert len(eng.generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0]) == 4
    assert eng.kv.rows and len(eng.kv.rows) == 1                                             # the second attention layer shares the first one's rows


def test_prefix_reuse_restores_state_and_rows():
    """State checkpoints: a second request with the same beginning starts behind it and generates the same text."""
    from fllm_b200.config import EngineConfig
    from fllm_b200.runtime.engine import LLMEngine
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    mc, weights = S.load_tensors(cfg, w, "cpu", torch.float32)
    ec = EngineConfig(dtype="fp32", max_num_seqs=2, num_kv_blocks=32, max_model_len=128, max_num_batched_tokens=64, state_cache_gb=0.1)
    eng = LLMEngine(mc, ec, device="cpu", weights=weights)
    p = S.prompt(cfg, 50, 3)
    sp = SamplingParams(max_tokens=5, ignore_eos=True)
    first = eng.generate([p], sp)
    assert eng.state_ckpt.stats["saved"] >= 1
    assert eng.generate([p], sp) == first and eng.state_ckpt.stats["restored"] >= 1
