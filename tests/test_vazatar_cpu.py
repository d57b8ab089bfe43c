"""Stack models without a GPU: configuration, converter, directory reader, page pool, trace replay and the scheduler's rules for recurrent
models (driven through a stand-in back end that computes with the plain implementation)."""
import io
import json

import pytest
import torch

import vazatar_models as M
import vazatar_oracle as O
from ollama_b200.convert.hf import convert_hf
from ollama_b200.engine.backend import make_backend, open_model
from ollama_b200.engine.cache import PAGE, CacheFull, PagedCache
from ollama_b200.engine.runner import CompletionRequest, Runner, RunnerOptions
from ollama_b200.engine.sampler import SamplingParams
from ollama_b200.engine.trace import replay
from ollama_b200.models.config import ModelConfig, config_from_gguf
from ollama_b200.models.stack import Rotation, parse_stack
from ollama_b200.models.weights import load_tensor


def test_rotation_frequencies_cover_the_three_branches():
    r = Rotation(16, 700.0, (4.0, 1.0, 3.0, 60.0))
    plain, got = Rotation(16, 700.0).freqs(), r.freqs()
    want = O.rotary_freqs(700.0, 16, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60})
    assert torch.allclose(torch.tensor(got, dtype=torch.float64), want, rtol=1e-14)
    ratio = [g / p for g, p in zip(got, plain)]
    assert ratio[0] == 1.0 and ratio[-1] == 0.25 and any(0.25 < x < 1.0 for x in ratio)


def test_layer_runs_follow_the_loop():
    for loop in (None, (0, 1, 1), (1, 3, 2), (2, 5, 3), (0, 5, 2)):
        cfg = M.config([M.mamba() for _ in range(5)], loop=loop)
        assert [(r.layer, r.joins) for r in parse_stack(cfg).runs()] == O.schedule(cfg)


def test_bad_configurations_are_refused():
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0].update(mlp={"kind": "other", "ff": 8}),
                   lambda c: c.update(loop={"start": 2, "stop": 2, "times": 1}), lambda c: c["layers"][0]["mixer"].update(kv_heads=2),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7)):
        cfg = json.loads(json.dumps(M.small()))
        change(cfg)
        with pytest.raises((ValueError, NotImplementedError)):
            parse_stack(cfg)


def test_directory_and_converted_file_hold_the_same_model(tmp_path):
    cfg = M.small()
    w = M.weights(cfg, 3)
    d = M.write(tmp_path / "ck", cfg, w)
    convert_hf(d, str(tmp_path / "m.gguf"))
    with open_model(d) as a, open_model(str(tmp_path / "m.gguf")) as b:
        ca, cb = config_from_gguf(a), config_from_gguf(b)
        assert ca.stack == cb.stack and ca.recurrent and ca.arch == "vazatar" and ca.vocab_size == cfg["vocab"]
        assert set(a.tensors) == set(b.tensors)
        for n in a.tensors:
            x, y = load_tensor(a, n), load_tensor(b, n)
            assert x.shape == y.shape and torch.equal(x.dequant(), y.dequant()), n
        assert torch.equal(load_tensor(a, "blk.0.attn_norm.weight").dequant(), w["l0.norm1"].float() + 1)
        assert torch.equal(load_tensor(a, "blk.1.ssm_out.weight").dequant(), w["l1.mix.o"].float())
        assert torch.allclose(load_tensor(a, "blk.1.ssm_a").dequant(), -torch.exp(w["l1.mix.A_log"].double()).float())
        with pytest.raises(NotImplementedError):
            make_backend(a, "cpu")


def test_unknown_tensor_is_an_error(tmp_path):
    cfg = M.small()
    w = M.weights(cfg, 3)
    w["l0.mix.extra"] = torch.zeros(3, dtype=torch.bfloat16)
    with pytest.raises(ValueError):
        open_model(M.write(tmp_path / "ck", cfg, w))


def test_cache_and_state_sizes():
    st = parse_stack(M.small())
    # runs: 0 | 1 2 1 2 | 3 4 (attention layers 0, 2, 2, 4)
    assert st.kv_bytes_per_token() == 2 * (1 * (40 + 24) + 2 * (2 * (12 + 32)) + 2 * (24 + 24))
    assert st.state_bytes() == 4 * (2 * 56 * (10 + 3) + 40 * (17 + 1))


def test_page_pool_reserves_releases_and_copies():
    c = PagedCache(3, 5 * PAGE, pool_tokens=6 * PAGE, device="cpu")
    t, s = c.add_pages(2, 4, torch.float32), c.add_state(7)
    c.reserve(0, 2 * PAGE + 1)
    c.reserve(1, PAGE)
    first = list(c.owned[0])
    c.reserve(0, 3 * PAGE)                    # nothing new, nothing moves
    assert c.owned[0] == first and len(c.free) == 2
    with pytest.raises(CacheFull):
        c.reserve(2, 3 * PAGE)                # more than the pool has left
    with pytest.raises(CacheFull):
        c.reserve(0, 5 * PAGE + 1)            # more than a slot can hold
    assert len(c.free) == 2 and c.owned[2] == []
    t[c.owned[0]] = torch.randn(3, 2, PAGE, 4)
    s[0] = 5.0
    c.release(1)
    c.copy(0, 1, 2 * PAGE + 1)
    assert not set(c.owned[0]) & set(c.owned[1])
    assert torch.equal(t[c.owned[0]], t[c.owned[1]]) and s[1, 0] == 5.0
    assert c.sync() > 0 and c.sync() == 0 and torch.equal(c.table[1, :3], torch.tensor(c.owned[1], dtype=torch.int32))
    c.release(0)
    assert sorted(c.free + c.owned[1]) == list(range(6))


class Plain:
    """Back end with the calls of a stack engine, computing with the plain implementation over the tokens each slot has seen."""
    name = "plain"
    supports_shift = False

    def __init__(self, cfg, w):
        self.raw, self.w = cfg, w
        self.cfg = ModelConfig(arch="vazatar", vocab_size=cfg["vocab"], stack=parse_stack(cfg))
        self.calls = []

    def alloc(self, n_slots, n_ctx, pool_tokens=None):
        self.n_slots, self.n_ctx = n_slots, n_ctx
        self.cache = PagedCache(n_slots, n_ctx, pool_tokens, "cpu")
        self.seen = [[] for _ in range(n_slots)]

    def step(self, segs, want):
        self.calls.append([len(t) for _, t, _ in segs])
        out = []
        for (slot, toks, p0), rows in zip(segs, want):
            self.cache.reserve(slot, p0 + len(toks))
            if p0 == 0:
                self.seen[slot] = []
            assert len(self.seen[slot]) == p0, "a recurrent state was asked to move back"
            self.seen[slot] = self.seen[slot] + list(toks)
            if rows:
                lg = O.forward(self.raw, self.w, self.seen[slot], torch.float32)
                out += [lg[p0 + r] for r in rows]
        return torch.stack(out) if out else None

    def prefill(self, slot, toks, pos0, need_logits=True, **_):
        r = self.step([(slot, toks, pos0)], [[len(toks) - 1] if need_logits else []])
        return r[0] if need_logits else None

    def prefill_many(self, segs, need):
        r = self.step(segs, [[len(t) - 1] if n else [] for (_, t, _), n in zip(segs, need)])
        it = iter(r if r is not None else [])
        return [next(it) if n else None for n in need]

    def decode(self, slots, toks, poss):
        return self.step([(s, [t], p) for s, t, p in zip(slots, toks, poss)], [[0]] * len(slots))

    def admit(self, slot, n, idle):
        dropped = []
        for s in [None, *idle]:
            if s is not None:
                self.cache.release(s)
                dropped.append(s)
            try:
                self.cache.reserve(slot, n)
                return True, dropped
            except CacheFull:
                pass
        return False, dropped

    def copy_rows(self, src, dst, n):
        assert n == len(self.seen[src])
        self.cache.copy(src, dst, n)
        self.seen[dst] = list(self.seen[src])

    def free_slot(self, slot):
        self.cache.release(slot)

    def weight_bytes(self):
        return 0

    kv_bytes = weight_bytes

    def close(self):
        pass


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(cfg, w, seq, torch.float32)[-1].argmax()))
    return seq[len(prompt):]


def collect(r, prompt, n, **kw):
    return r.submit(CompletionRequest(prompt=prompt, sampling=SamplingParams(temperature=0), num_predict=n, ignore_eos=True, **kw))


def drain(seq):
    out = []
    while True:
        ch = seq.out.get(timeout=60)
        assert not ch.error, ch.error
        out += ch.tokens
        if ch.done:
            return out, ch


@pytest.fixture(scope="module")
def tiny():
    cfg = M.config([M.attention(ff=None), M.mamba(ff=24)], loop=None, width=24, vocab=61)
    return cfg, M.weights(cfg, 5)


def test_scheduler_mixes_prompts_with_running_sequences(tiny):
    cfg, w = tiny
    be = Plain(cfg, w)
    r = Runner(None, RunnerOptions(num_ctx=96, num_parallel=3, num_batch=7), backend=be)
    try:
        prompts = [M.tokens(n, cfg["vocab"], n) for n in (3, 25, 18, 9, 31)]
        seqs = [collect(r, p, 6) for p in prompts]
        assert [drain(s)[0] for s in seqs] == [greedy(cfg, w, p, 6) for p in prompts]
        assert any(1 in c and max(c) > 1 for c in be.calls) and r.stats.get("mixed_steps", 0) > 0
        assert all(sum(c) <= 7 + 3 for c in be.calls)
    finally:
        r.close()


def test_scheduler_reuses_a_recurrent_prefix_only_as_a_whole(tiny):
    cfg, w = tiny
    be = Plain(cfg, w)
    r = Runner(None, RunnerOptions(num_ctx=128, num_parallel=2), backend=be)
    try:
        p = M.tokens(20, cfg["vocab"], 1)
        out, _ = drain(collect(r, p, 5))
        held = p + out[:-1]                       # what the slot's state has seen
        longer = held + M.tokens(6, cfg["vocab"], 2)
        got, ch = drain(collect(r, longer, 4))
        assert ch.cached_tokens == len(held) and got == greedy(cfg, w, longer, 4)
        branch = p[:12] + M.tokens(9, cfg["vocab"], 3)      # shares a prefix, but the state is past it
        got, ch = drain(collect(r, branch, 4))
        assert ch.cached_tokens == 0 and got == greedy(cfg, w, branch, 4)
    finally:
        r.close()


def test_scheduler_waits_for_pages_and_uses_them_again(tiny):
    cfg, w = tiny
    be = Plain(cfg, w)
    r = Runner(None, RunnerOptions(num_ctx=2 * PAGE, num_parallel=4, kv_pool_tokens=3 * PAGE), backend=be)
    try:
        prompts = [M.tokens(n, cfg["vocab"], 50 + n) for n in (70, 20, 66, 30, 64)]      # two pages, one page, two pages, ...
        seqs = [collect(r, p, 3) for p in prompts]
        assert [drain(s)[0] for s in seqs] == [greedy(cfg, w, p, 3) for p in prompts]
    finally:
        r.close()


def test_context_shift_evaluates_the_kept_tokens_again(tiny):
    cfg, w = tiny
    r = Runner(None, RunnerOptions(num_ctx=24), backend=Plain(cfg, w))
    try:
        out, ch = drain(collect(r, M.tokens(15, cfg["vocab"], 9), 20, num_keep=4))
        assert len(out) == 20 and r.stats["context_shifts"] >= 1
    finally:
        r.close()


def test_trace_replay_batches_resumes_and_frees(tiny, tmp_path):
    cfg, w = tiny
    be = Plain(cfg, w)
    be.alloc(4, 2 * PAGE, 2 * PAGE)
    a, b, c = (M.tokens(n, cfg["vocab"], 70 + n) for n in (40, 9, 100))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [2, 6]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:], "want": [5, 0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[7:], "want": [32]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c, "want": []}], "end": ["c"]}]
    said = []
    replay(be, io.StringIO("\n".join(json.dumps(s) for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)] and len(be.cache.free) == be.cache.n_pages
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "1.f32", "2.f32"]
    la, lb = O.forward(cfg, w, a, torch.float32), O.forward(cfg, w, b, torch.float32)
    import numpy as np
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
    assert torch.allclose(read(0), la[[2, 6]], atol=1e-4) and torch.allclose(read(1), lb[[8, 3]], atol=1e-4) and torch.allclose(read(2), la[39:], atol=1e-4)
