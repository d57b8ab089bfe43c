"""The Kavenex design without a GPU: its plain implementation, configuration, converter, directory reader, and the scheduler with a stand-in
back end that computes with the plain implementation."""
import io
import json
import math

import pytest
import torch

import kavenex_models as M
import kavenex_oracle as O
from ollama_b200.convert.hf import convert_hf
from ollama_b200.engine.backend import make_backend, open_model
from ollama_b200.engine.cache import PagedCache
from ollama_b200.engine.runner import CompletionRequest, Runner, RunnerOptions
from ollama_b200.engine.sampler import SamplingParams
from ollama_b200.engine.trace import replay
from ollama_b200.models.config import ModelConfig, config_from_gguf
from ollama_b200.models.stack import DenseMLP, ExpertMLP, LatentMixer, parse_stack
from ollama_b200.models.weights import load_tensor


# -- the plain implementation against identities it must satisfy ------------------------------------------------
def test_rotation_turns_neighbouring_pairs_and_keeps_relative_angles():
    x = torch.randn(9, 2, 6, dtype=O.F64)
    pos = torch.arange(9)
    y = O.rotate_pairs(x, pos, 30.0)
    assert torch.equal(y[0], x[0])
    assert torch.allclose(y[..., 0::2] ** 2 + y[..., 1::2] ** 2, x[..., 0::2] ** 2 + x[..., 1::2] ** 2)
    a = 4 * 30.0 ** (-2.0 / 6)
    assert torch.allclose(y[4, 1, 2], x[4, 1, 2] * math.cos(a) - x[4, 1, 3] * math.sin(a))
    q, k = (x[:1, 0].expand(9, -1)[:, None], x[1:2, 0].expand(9, -1)[:, None])
    d = O.rotate_pairs(q, pos, 30.0)[:, 0] @ O.rotate_pairs(k, pos, 30.0)[:, 0].t()
    assert torch.allclose(d[5, 3], d[7, 5]) and not torch.allclose(d[5, 3], d[5, 4])


def test_layer_norm_centres_and_scales():
    x = torch.randn(4, 30, dtype=O.F64) * 3 + 5
    y = O.layer_norm(x, torch.ones(30), torch.zeros(30), 0.0)
    assert y.mean(-1).abs().max() < 1e-12 and (y.var(-1, unbiased=False) - 1).abs().max() < 1e-9
    assert torch.allclose(O.layer_norm(x, torch.full((30,), 2.0), torch.full((30,), 3.0), 0.0), 2 * y + 3)


def test_router_weights_are_a_softmax_over_the_chosen_and_biases_count():
    h = torch.randn(20, 8, dtype=O.F64)
    w = torch.randn(5, 8, dtype=O.F64)
    idx, wt = O.route(h, w, torch.tensor([0.0, 0, 0, 0, 100.0]), 2)
    assert (idx[:, 0] == 4).all() and torch.allclose(wt.sum(-1), torch.ones(20, dtype=O.F64))
    idx, wt = O.route(h, w, torch.zeros(5), 5)
    assert torch.allclose(wt, torch.softmax(h @ w.t(), -1).gather(1, idx))


def test_expert_limits():
    one = torch.ones(1, 1, dtype=O.F64)
    y = [O.expert(torch.full((1, 1), v, dtype=O.F64), one, one, one, 2.0).item() for v in (-9.0, 2.0, 9.0)]
    s = 1 / (1 + math.exp(-1.702 * 2))
    assert y[1] == pytest.approx(2 * s * 3) and y[2] == pytest.approx(y[1])
    assert y[0] == pytest.approx(-9.0 / (1 + math.exp(1.702 * 9)) * (-2 + 1))       # the gate has no lower limit


def test_a_later_token_changes_nothing_before_it():
    cfg = M.small()
    w = M.weights(cfg, 5)
    t = M.tokens(20, cfg["vocab"], 1)
    a, b = O.forward(cfg, w, t), O.forward(cfg, w, t[:12] + M.tokens(8, cfg["vocab"], 2))
    assert torch.allclose(a[:12], b[:12]) and not torch.allclose(a[12:], b[12:])


# -- configuration, names, files --------------------------------------------------------------------------------
def test_configuration():
    st = parse_stack(M.small())
    assert [type(L.mixer) for L in st.layers] == [LatentMixer] * 5 and not st.design.parallel and st.residual_mult == 0.6 and st.side_dim == 12
    assert [type(L.mlp) for L in st.layers] == [DenseMLP, ExpertMLP, DenseMLP, type(None), ExpertMLP]
    assert st.layers[1].mlp.shared.limit == 0.9 and st.layers[4].mlp.shared is None and st.layers[0].mlp.gated
    assert [(r.layer, r.joins) for r in st.runs()] == O.schedule(M.small())
    assert [r.turn for r in st.runs() if r.joins] == [0, 1]
    # runs: 0 | 1 2 1 2 | 3 4
    assert st.kv_bytes_per_token() == 2 * (3 * (36 + 8) + 2 * (24 + 16) + 2 * (50 + 2)) and st.state_bytes() == 0 and not st.recurrent
    bare = parse_stack({k: v for k, v in M.config([M.layer()], loop=None).items() if k not in ("residual_mult", "token_side", "embedding", "loop")})
    assert bare.residual_mult == 1.0 and bare.side_dim == 0 and bare.embed_scale == 1.0 and bare.loop is None
    unlimited = M.moe()
    del unlimited["expert"]["limit"]
    assert parse_stack(M.config([M.layer(unlimited)], loop=None)).layers[0].mlp.expert.limit == math.inf


def test_bad_configurations_are_refused():
    for change in (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), lambda c: c["layers"][1]["mlp"].update(kind="other"),
                   lambda c: c.update(loop={"start": 2, "stop": 6, "times": 1}), lambda c: c["layers"][0]["mixer"].update(rot_dim=7)):
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
        assert ca.stack == cb.stack == parse_stack(cfg) and ca.arch == "kavenex" and ca.vocab_size == cfg["vocab"] and ca.n_experts == 9
        assert set(a.tensors) == set(b.tensors)
        for n in a.tensors:
            x, y = load_tensor(a, n), load_tensor(b, n)
            assert x.shape == y.shape and torch.equal(x.dequant(), y.dequant()), n

        def get(n):
            return load_tensor(b, n).dequant()
        assert torch.equal(get("blk.0.attn_norm.weight"), w["l0.norm1"].float()) and torch.equal(get("blk.0.attn_norm.bias"), w["l0.norm1.b"].float())
        assert torch.equal(get("blk.1.ffn_up_exps.weight"), torch.stack([w[f"l1.mlp.e{e}.up"].float() for e in range(6)]))
        assert torch.equal(get("blk.1.ffn_gate_shexp.weight"), w["l1.mlp.shared.gate"].float())
        assert torch.equal(get("per_layer_token_embd.weight"), w["side.embed"].float())
        with pytest.raises(NotImplementedError):
            make_backend(a, "cpu")


def test_missing_and_unknown_tensors_are_errors(tmp_path):
    cfg = M.small()
    for name, change in (("l1.mlp.e5.up", "drop"), ("l0.mix.extra", "add"), ("l1.mlp.e6.up", "add")):
        w = M.weights(cfg, 3)
        if change == "drop":
            del w[name]
        else:
            w[name] = torch.zeros(3, 3, dtype=torch.bfloat16)
        with pytest.raises(ValueError):
            open_model(M.write(tmp_path / name, cfg, w))


def test_memory_estimate_counts_latents():
    from ollama_b200.convert.stack import stack_kv
    from ollama_b200.server.sched import predict_memory

    class Model:
        size = 1000

        def kv(self):
            return stack_kv(M.small(), "m")
    assert predict_memory(Model(), 100, 2) == 1000 + 2 * 100 * parse_stack(M.small()).kv_bytes_per_token()


# -- scheduler and trace replay over a stand-in back end -----------------------------------------------------------
class Plain:
    """Back end with the calls of a stack engine, computing with the plain implementation over the tokens each slot has seen."""
    name = "plain"
    supports_shift = False

    def __init__(self, cfg, w):
        self.raw, self.w = cfg, w
        self.cfg = ModelConfig(arch="kavenex", vocab_size=cfg["vocab"], stack=parse_stack(cfg))

    def alloc(self, n_slots, n_ctx, pool_tokens=None):
        self.n_slots, self.n_ctx = n_slots, n_ctx
        self.cache = PagedCache(n_slots, n_ctx, pool_tokens, "cpu")
        self.seen = [[] for _ in range(n_slots)]

    def step(self, segs, want):
        rows = []
        for (slot, toks, p0), w in zip(segs, want):
            self.cache.reserve(slot, p0 + len(toks))
            self.seen[slot] = self.seen[slot][:p0] + list(toks)
            assert len(self.seen[slot]) == p0 + len(toks)
            if len(w):
                rows.append(O.forward(self.raw, self.w, self.seen[slot])[[p0 + int(j) for j in w]])
        return torch.cat(rows).float() if rows else None

    def prefill(self, slot, tokens, pos0, need_logits=True):
        out = self.step([(slot, tokens, pos0)], [[len(tokens) - 1] if need_logits else []])
        return out[0] if need_logits else None

    def prefill_many(self, segs, need_logits):
        return [self.prefill(s, t, p, n) for (s, t, p), n in zip(segs, need_logits)]

    def decode(self, slots, tokens, positions):
        return self.step([(s, [t], p) for s, t, p in zip(slots, tokens, positions)], [[0]] * len(slots))

    def copy_rows(self, src, dst, n):
        self.cache.copy(src, dst, n)
        self.seen[dst] = self.seen[src][:n]

    def admit(self, slot, n_tokens, idle):
        from ollama_b200.engine.stack import StackBackend
        return StackBackend.admit(self, slot, n_tokens, idle)

    def free_slot(self, slot):
        self.cache.release(slot)
        self.seen[slot] = []

    def weight_bytes(self):
        return 0

    kv_bytes = weight_bytes

    def close(self):
        pass


def test_greedy_generation_and_prefix_reuse_through_the_runner():
    cfg = M.config([M.layer(M.dense(16), kv_rank=12), M.layer(M.moe(4, 2, 8), kv_rank=12)], loop=(0, 1, 2), width=24, vocab=41)
    w = M.weights(cfg, 9)
    r = Runner(None, RunnerOptions(num_ctx=96, num_parallel=2, num_batch=16, kv_pool_tokens=3 * 64), backend=Plain(cfg, w))

    def greedy(prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(O.forward(cfg, w, seq)[-1].argmax()))
        return seq[len(prompt):]
    try:
        def ask(p, n):
            chunks = list(r.completion(CompletionRequest(prompt=p, sampling=SamplingParams(temperature=0), num_predict=n, ignore_eos=True)))
            return [t for c in chunks for t in c.tokens], chunks[-1].cached_tokens
        p = M.tokens(21, cfg["vocab"], 1)
        got, _ = ask(p, 5)
        assert got == greedy(p, 5)
        other = p[:15] + M.tokens(6, cfg["vocab"], 2)          # branches inside the prompt: no recurrent state, so the common part is reused
        got, cached = ask(other, 4)
        assert got == greedy(other, 4) and cached == 15
    finally:
        r.close()


def test_replay_of_a_trace(tmp_path):
    import numpy as np
    cfg = M.config([M.layer(M.dense(16))], loop=(0, 1, 2), width=24, vocab=41)
    w = M.weights(cfg, 9)
    be = Plain(cfg, w)
    be.alloc(4, 128, 256)
    a = M.tokens(9, cfg["vocab"], 1)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:4], "want": [1, 3]}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": a[4:], "want": [4]}], "end": ["x"]}]
    said = []
    replay(be, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    full = O.forward(cfg, w, a).float().numpy()
    assert said == ["done 0", "done 1"]
    assert np.allclose(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1), full[[1, 3]], atol=1e-5)
    assert np.allclose(np.fromfile(tmp_path / "1.f32", "<f4"), full[8], atol=1e-5)
    assert len(be.cache.free) == be.cache.n_pages
