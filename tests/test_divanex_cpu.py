"""Divanex through the engine on the CPU (PyTorch operators) against the plain statement in tests/divanex_oracle.py:
configuration and loading, schedules, pages and state rows that are used again, generation."""
import copy
import dataclasses
import math

import pytest
import torch

import divanex_cases as S
import divanex_oracle as O
from fllm_b200.config import EngineConfig, ModelConfig, ParallelConfig, preset
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
    for name in ("odd", "wide-heads"):
        cfg, w, toks, want = S.expected(name, 41, 1)
        assert S.error(S.feed(S.TraceReplay(S.engine(cfg, w, f32=False)), "a", toks, [7]), want) < 8e-2


def test_a_far_token_shows_in_the_logits():
    """The weights are sharp enough for the other tests to mean something: the last logits move far beyond the tolerances when
    one early token changes, with attention only (a lost key) and with recurrent layers only (a lost state)."""
    for name in ("attention-only", "mamba-only", "odd"):
        cfg, w, toks, want = S.expected(name, 41, 1)
        for place in (0, 7, 16):
            other = list(toks)
            other[place] = (other[place] + 11) % cfg["vocab"]
            assert S.error(O.forward(cfg, w, other, torch.float64)[-1:], want[-1:]) > 50 * TOL, (name, place)


@pytest.mark.parametrize("change", ["postln_alpha", "logit_scale", "embedding", "softcap", "coef", "every", "scale", "limit", "norm_groups", "eps", "side"])
def test_every_constant_is_read_from_the_configuration(change):
    """Another value of one constant: the engine follows the oracle, and the logits move."""
    # (attention in front, its norms and the norm behind the sum are blind to the embedding's scale)
    base, w, toks, want = S.expected("mamba-only" if change == "embedding" else "odd", 41, 1)
    cfg = copy.deepcopy(base)
    first, second = cfg["layers"][0], cfg["layers"][1]
    if change in ("postln_alpha", "logit_scale"):
        cfg[change] *= 1.5
    elif change == "embedding":
        cfg["embedding"]["scale"] = 0.5
    elif change in ("softcap", "scale"):
        first["mixer"][change] *= 0.4
    elif change == "coef":
        first["mixer"]["q_temp"]["coef"] = 0.9
    elif change == "every":
        first["mixer"]["q_temp"]["every"] = 3
    elif change == "limit":
        second["mlp"]["limit"] = 0.3
    elif change == "norm_groups":
        second["mixer"]["norm_groups"] = 1
    elif change == "eps":
        cfg["norm"]["eps"] = 0.05
    else:                                                # another layer's slice of the token table
        w = dict(w, **{"side.embed": w["side.embed"].roll(cfg["token_side"]["dim"], 1)})
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


def test_generation_through_the_scheduler():
    """Greedy text of unequal requests with chunked prompts: each token is the oracle's best one."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, chunk=16, seqs=3, spare=4)
    prompts = [S.prompt(cfg, n, n) for n in (3, 40, 17, 9)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = O.forward(cfg, w, p + o, torch.float64)[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert len(o) == 8 and float(gap.max()) < 1e-4 * float(lg.std())


def test_prefix_blocks_are_shared_without_recurrent_layers():
    """An attention-only model reuses cached prompt blocks, rows and factors."""
    cfg = S.CONFIGS["attention-only"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w)
    eng = LLMEngine(eng.model_cfg, dataclasses.replace(eng.cfg, enable_prefix_caching=True), device="cpu", weights=eng.weights)
    p, sp = S.prompt(cfg, 40, 3), SamplingParams(max_tokens=4, ignore_eos=True)
    first = eng.generate([p], sp)
    before = eng.stats.prefill_tokens
    assert eng.generate([p], sp) == first and eng.stats.prefill_tokens - before < 20


def test_checkpoint_directory_and_config(tmp_path):
    cfg, w, toks, want = S.expected("odd", 41, 1)
    mc, weights, tok = S.load_model(S.write_checkpoint(tmp_path / "m", cfg, w), "cpu", dtype=torch.float32)
    assert tok is None and mc.arch == "divanex" and mc.native_f32 and mc.native_part == "tied" and mc.has_recurrent and mc.has_row_cache
    assert [mc.layer_kind(i) for i in range(4)] == ["tied", "mamba2", "tied", "mamba2"] and [mc.ffn_kind(i) for i in range(4)] == ["glu", "glu", "none", "none"]
    assert ModelConfig.from_dict(mc.to_dict()) == mc
    from fllm_b200.models.row_cache import RowCache, RowSpec
    specs = RowCache.specs(mc, range(4))
    assert specs == [RowSpec(64, 2), RowSpec(64, 5)] and RowCache.bytes_per_block(specs, 16) == 16 * 7 * (128 + 4)
    assert weights.nbytes() > sum(t.numel() for t in w.values()) * 4
    bad = dict(w)
    bad["l1.mix.in"] = bad["l1.mix.in"][:-1]
    with pytest.raises(ValueError):
        S.load_tensors(cfg, bad, "cpu", torch.float32)
    for key, value in (("vdim", 21), ("kv_heads", 4)):
        broken = copy.deepcopy(cfg)
        broken["layers"][0]["mixer"][key] = value
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(broken)
    broken = copy.deepcopy(cfg)
    broken["layers"][1]["type"] = "other"
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(broken)


def test_preset_runs_with_random_weights():
    eng = LLMEngine(preset("divanex-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64, max_num_seqs=2), device="cpu")
    out = eng.generate([[1, 2, 3], [4, 5]], SamplingParams(max_tokens=5, ignore_eos=True))
    assert [len(o) for o in out] == [5, 5]
    eng = LLMEngine(preset("divanex-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64, max_num_seqs=2), device="cpu")
    assert out == eng.generate([[1, 2, 3], [4, 5]], SamplingParams(max_tokens=5, ignore_eos=True))


def test_tensor_parallel_ranks_are_refused():
    with pytest.raises(NotImplementedError):
        LLMEngine(preset("divanex-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64), ParallelConfig(tp=2), device="cpu")


def test_query_temperature_steps_exactly_at_its_multiples():
    from fllm_b200.ops.reference import RefOps
    pos = torch.tensor([0, 5, 8, 9, 18, 19, 99, 100], dtype=torch.int32)
    x = torch.ones(8, 16)
    cache, factor = torch.zeros(1, 1, 16, 64), torch.zeros(1, 1, 16)
    _, qf = RefOps().tied_prepare(x, 8, 1, 8, pos, torch.arange(8, dtype=torch.int32), -1.0, 2.0, 0.5, 10.0, cache, factor)
    want = [2 * (1 + 0.5 * math.log((p + 1) // 10 + 1)) for p in pos.tolist()]
    assert torch.allclose(qf[:, 0], torch.tensor(want), rtol=1e-6)
