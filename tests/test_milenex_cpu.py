"""Milenex through the engine on the CPU (PyTorch operators) against the plain statement in tests/milenex_oracle.py: configuration
and loading, schedules, pages and state rows that are used again, generation."""
import copy

import pytest
import torch

import milenex_cases as S
import milenex_oracle as O
from fllm_b200.config import EngineConfig, ModelConfig, MoeSpec, ParallelConfig, preset
from fllm_b200.models.moe import route_reference
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
        assert S.error(S.feed(S.TraceReplay(S.engine(cfg, w, f32=False)), "a", toks, [7]), want) < 6e-2


def test_a_token_in_reach_shows_in_the_logits():
    """The weights are sharp enough for the other tests to mean something: the last logits move far beyond the tolerances when a token
    inside the reach of a window, of a convolution or of the token shift changes, and not at all when one outside it does."""
    one = {"window": S.config([S.rotary(2, 1, 8, 8, 20, 4, 1)], 61, 40), "distance": S.config([S.talking(2, 2, 8, 8, 20)], 61, 40),
           "conv": S.config([S.rotary(2, 1, 8, 8, 1, 4, 4)], 61, 40), "shift": S.config([S.talking(1, 1, 8, 8, 1)], 61, 40)}
    reach = {"window": 21, "distance": 21, "conv": 5, "shift": 2}                            # the shift adds a token to each
    for name, cfg in one.items():
        w, toks = S.tensors(cfg), S.prompt(cfg, 41, 2)
        want = O.forward(cfg, w, toks, torch.float64)[-1:]
        for back in (0, 1, reach[name] - 1, reach[name]):
            other = list(toks)
            other[40 - back] = (other[40 - back] + 11) % cfg["vocab"]
            moved = S.error(O.forward(cfg, w, other, torch.float64)[-1:], want)
            assert moved > 50 * TOL if back < reach[name] else moved == 0, (name, back, moved)


CHANGES = {
    "window": lambda c: c["layers"][0]["mixer"]["mask"].update(size=18), "window_2": lambda c: c["layers"][1]["mixer"]["mask"].update(size=25),
    "scale": lambda c: c["layers"][0]["mixer"].update(scale=0.1), "scale_2": lambda c: c["layers"][1]["mixer"].update(scale=0.3),
    "base": lambda c: c["layers"][0]["mixer"]["rot"].update(base=40.0), "rot_dims": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=20),
    "no_rot": lambda c: c["layers"][2]["mixer"]["rot"].update(dims=0), "top": lambda c: c["layers"][0]["mlp"]["router"].update(top=2),
    "keep": lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3), "count": lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=2),
    "no_groups": lambda c: c["layers"][0]["mlp"]["router"].pop("groups"), "limit": lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.3),
    "shared_limit": lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.2), "no_shared": lambda c: c["layers"][0]["mlp"].pop("shared"),
    "eps": lambda c: c["norm"].update(eps=0.3), "no_mlp": lambda c: c["layers"][1].update(mlp=None), "times": lambda c: c["loop"].update(times=2),
    "start": lambda c: c["loop"].update(start=0), "stop": lambda c: c["loop"].update(stop=4), "no_loop": lambda c: c.update(loop=None),
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


def test_every_tensor_is_read():
    """Scaling any tensor moves the logits of the engine as it moves those of the oracle."""
    cfg, w, toks, want = S.expected("odd", 24, 1)
    seen = set()
    for name in w:
        kind = ".".join(x for x in name.split(".") if not (x[0] in "le" and x[1:].isdigit()))
        key = (kind, cfg["layers"][int(name.split(".")[0][1:])]["type"] if name[0] == "l" and name[1].isdigit() else "")
        if key in seen:
            continue
        seen.add(key)
        other = dict(w, **{name: (w[name].float() * 1.5 + 0.1).bfloat16()})
        moved = O.forward(cfg, other, toks, torch.float64)
        if ".e" not in name:                               # (an expert may go unused)
            assert S.error(moved, want) > 20 * TOL, name
        assert S.error(S.feed(S.TraceReplay(S.engine(cfg, other)), "a", toks, [5, 20]), moved) < TOL, name
    assert len(seen) > 30


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


def _best(cfg, w, prompts, outs, n):
    for p, o in zip(prompts, outs):
        lg = O.forward(cfg, w, p + o, torch.float64)[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert len(o) == n and float(gap.max()) < 1e-4 * float(lg.std())


def test_generation_through_the_scheduler_gives_back_pages_behind_the_windows():
    """Greedy text of unequal requests with chunked prompts in a pool that is too small for whole sequences: each token is the
    oracle's best one, and the pages no window reaches any more are used again."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, chunk=16, seqs=2, spare=4, blocks=10)
    assert eng.scheduler.window == 33
    prompts = [S.prompt(cfg, n, n) for n in (3, 75, 17, 60)]
    _best(cfg, w, prompts, eng.generate(prompts, SamplingParams(max_tokens=30, ignore_eos=True)), 30)


def test_padding_rows_of_a_captured_step_point_at_a_real_block():
    """Rows that fill a decode step up to its captured size have one key, the first of block 0, whatever the staging buffer held:
    entries of sequences whose first pages fell behind the window (-1) stay out of them."""
    cfg = S.CONFIGS["odd"]
    eng = S.engine(cfg, S.tensors(cfg), chunk=16, seqs=4, spare=4, blocks=48)
    build, seen = eng._build_batch, []

    def checked(step, pad_to=0, slot=0):
        if step.all_decode:
            n, b = len(step.seqs), build(step, pad_to=4, slot=slot)
            t = b.block_tables
            seen.append((n, int((t[:n, 0] < 0).sum())))
            assert t.shape[0] == 4 and t[n:, 0].tolist() == [0] * (4 - n)
            assert b.row_seq.tolist() == list(range(4)) and b.seq_lens[n:].tolist() == [1] * (4 - n) and b.slots[n:].tolist() == [-1] * (4 - n)
            assert b.seq_state[n:].tolist() == [eng.rstate.slots - 1] * (4 - n)
        return build(step, pad_to=pad_to, slot=slot)

    eng._build_batch = checked
    for k, n in enumerate((60, 64, 55, 58)):
        eng.add_request(S.prompt(cfg, n, n), SamplingParams(max_tokens=24 + 4 * k, ignore_eos=True))
    while eng.scheduler.has_work():
        eng.step()
    assert any(pruned for _, pruned in seen) and {n for n, _ in seen} == {1, 2, 3, 4}      # pruned first pages, then fewer and fewer sequences


def test_a_cached_prefix_restores_the_states():
    """Prompts that share a prefix: the later ones continue from kept copies of the shift and convolution rows."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, chunk=32, seqs=2, spare=4, enable_prefix_caching=True, state_cache_gb=0.1)
    shared = S.prompt(cfg, 64, 3)
    for tail in (5, 9, 30):
        p = shared + S.prompt(cfg, tail, tail)
        _best(cfg, w, [p], eng.generate([p], SamplingParams(max_tokens=6, ignore_eos=True)), 6)
    assert eng.state_ckpt.stats["restored"] >= 1


def test_checkpoint_directory_and_config(tmp_path):
    cfg, w, toks, want = S.expected("odd", 41, 1)
    mc, weights, tok = S.load_model(S.write_checkpoint(tmp_path / "m", cfg, w), "cpu", dtype=torch.float32)
    assert tok is None and mc.arch == "milenex" and mc.native_f32 and mc.native_part == "maps" and mc.has_recurrent and mc.has_row_cache
    assert mc.layer_source == [0, 1, 2, 1, 2, 1, 2, 3] and mc.embed_again == [3, 5] and mc.num_layers == 8 == len(weights.layers)
    assert weights.layers[1] is weights.layers[3] and weights.layers[2] is weights.layers[6] and weights.layers[0] is not weights.layers[1]
    assert [mc.ffn_kind(i) for i in range(8)] == ["moe", "plain", "none", "plain", "none", "plain", "none", "moe"]
    assert ModelConfig.from_dict(mc.to_dict()) == mc
    assert mc.moe_of(0) == MoeSpec(6, 3, "deepseek_v2", groups=3, topk_groups=2, act="swiglu_oai", fp32_router=True, masked=float("-inf"), limit=0.8, shared_limit=0.5)
    from fllm_b200.models.recurrent import RecurrentState
    from fllm_b200.models.row_cache import RowCache, RowSpec
    specs = RowCache.specs(mc, range(8))
    assert specs[0] == RowSpec(64, 2, 64, 2) and specs[1] == specs[3] == RowSpec(64, 3, 64, 1) and specs[7] == RowSpec(64, 1, 64, 1)
    conv = {0: 2 * (120 + 40 + 56), 2: 4 * (40 + 16 + 8)}                                    # taps - 1 rows of the padded projections
    assert RecurrentState.bytes_per_slot(mc, range(8)) == 8 * 80 * 4 + 2 * (conv[0] + 3 * conv[2])
    assert RecurrentState(mc, range(8), 3, "cpu").nbytes() == 3 * RecurrentState.bytes_per_slot(mc, range(8))
    bad = dict(w)
    bad["l1.mix.talk"] = bad["l1.mix.talk"][:-1]
    with pytest.raises(ValueError):
        S.load_tensors(cfg, bad, "cpu", torch.float32)
    breaks = [lambda c: c["layers"][0]["mixer"].update(kv_heads=4), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), lambda c: c["layers"][1].update(type="other"),
              lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
              lambda c: c["layers"][0]["mixer"].update(conv=9), lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["loop"].update(stop=5),
              lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), lambda c: c["layers"][1]["mlp"].update(kind="other")]
    for change in breaks:
        broken = copy.deepcopy(cfg)
        change(broken)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(broken)


def test_residual_after_every_layer():
    """The engine's residual of a model cut behind each of its layers."""
    base, w, toks, _ = S.expected("tensor-cores", 41, 1)
    base = dict(base, loop=dict(start=0, stop=2, times=2))
    for n in range(2, len(base["layers"]) + 1):
        cut, want = dict(base, layers=base["layers"][:n]), []
        tensors = dict(w, **{"final.norm": torch.zeros(base["width"]), "head": torch.eye(base["vocab"], base["width"])})
        O.forward(cut, tensors, toks, torch.float64, want)
        assert len(want) == n + 2
        eng = S.engine(cut, tensors)
        eng.decoder.capture_hidden = True
        S.feed(S.TraceReplay(eng), "a", toks, [])
        got = eng.decoder.last_hidden.double()[:, :base["width"]]
        assert float((got - O.rms(want[-1], base["norm"]["eps"])).abs().max()) < 1e-4, n


@pytest.mark.parametrize("E,count,keep,top", [(12, 4, 2, 3), (6, 6, 3, 2), (8, 2, 1, 4), (5, 1, 1, 5)])
def test_experts_are_chosen_inside_the_best_groups(E, count, keep, top):
    """Choice scores below zero: experts outside the kept groups stay out, which a mask of zero would get wrong."""
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(40, E, generator=g), torch.randn(E, generator=g) * 0.3 - 1.5
    ids, wts = route_reference(MoeSpec(E, top, "deepseek_v2", groups=count, topk_groups=keep, masked=float("-inf"), fp32_router=True), z, corr)
    s = torch.softmax(z, -1)
    for t in range(40):
        want = O.choose(s[t], corr, top, count, keep)
        assert ids[t].tolist() == want and torch.allclose(wts[t], s[t, want])


def test_preset_runs_with_random_weights():
    run = lambda: LLMEngine(preset("milenex-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64, max_num_seqs=2), device="cpu").generate(
        [[1, 2, 3], [4, 5]], SamplingParams(max_tokens=5, ignore_eos=True))
    out = run()
    assert [len(o) for o in out] == [5, 5] and out == run()


def test_tensor_parallel_ranks_are_refused():
    with pytest.raises(NotImplementedError):
        LLMEngine(preset("milenex-tiny"), EngineConfig(num_kv_blocks=16, max_model_len=64), ParallelConfig(tp=2), device="cpu")
