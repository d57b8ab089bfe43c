"""The Tirudra design without a GPU: its plain implementation, configuration, converter, directory reader, and the scheduler with a stand-in
back end that computes with the plain implementation."""
import io
import json
import math

import pytest
import torch

import test_vazatar_cpu as V
import tirudra_models as M
import tirudra_oracle as O
from ollama_b200.convert.hf import convert_hf
from ollama_b200.engine.backend import make_backend, open_model
from ollama_b200.engine.cache import PAGE
from ollama_b200.engine.runner import CompletionRequest, Runner, RunnerOptions
from ollama_b200.engine.sampler import SamplingParams
from ollama_b200.engine.trace import replay
from ollama_b200.models.config import ModelConfig, config_from_gguf
from ollama_b200.models.stack import AttentionMixer, ExpertMLP, Mamba2Mixer, Rotation, parse_stack
from ollama_b200.models.weights import load_tensor


# -- the plain implementation against identities it must satisfy ------------------------------------------------
def test_window_and_kept_tokens():
    ok = O.window_visible(12, 3, 2)
    assert [j for j in range(12) if ok[9, j]] == [0, 1, 7, 8, 9]
    assert [j for j in range(12) if ok[1, j]] == [0, 1] and [j for j in range(12) if ok[3, j]] == [0, 1, 2, 3]
    assert torch.equal(O.window_visible(5, 1, 0), torch.eye(5).bool()) and torch.equal(O.window_visible(5, 5, 0), O.window_visible(5))


def test_scan_is_the_sum_over_earlier_tokens():
    g = torch.Generator().manual_seed(1)
    T, H, p, n, G = 7, 4, 3, 5, 2

    def r(*s):
        return torch.randn(*s, generator=g, dtype=O.F64)
    x, dt, a, B, C, D = r(T, H, p), r(T, H).abs(), -r(H).abs(), r(T, G, n), r(T, G, n), r(H)
    y = O.ssd_scan(x, dt, a, B, C, D)
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + torch.exp(a[h] * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (B[s, h // 2] @ C[t, h // 2]) * x[s, h]
            assert torch.allclose(y[t, h], want)


def test_convolution_and_group_norm():
    u, w = torch.randn(6, 2, dtype=O.F64), torch.randn(2, 3, dtype=O.F64)
    y = O.short_conv(u, w)
    assert torch.allclose(y[0], w[:, 2] * u[0]) and torch.allclose(y[4], w[:, 0] * u[2] + w[:, 1] * u[3] + w[:, 2] * u[4])
    x, z = torch.randn(3, 12, dtype=O.F64), torch.randn(3, 12, dtype=O.F64)
    n = O.gated_group_norm(x, z, torch.ones(12), 3, 0.0)
    assert torch.allclose((n.view(3, 3, 4) ** 2).mean(-1), torch.ones(3, 3, dtype=O.F64))
    assert not torch.allclose(n / n[:, :1], (x * O.silu(z)) / (x * O.silu(z))[:, :1])      # parts have scales of their own
    assert torch.allclose(n[:, :4] / n[:, :1], (x * O.silu(z))[:, :4] / (x * O.silu(z))[:, :1])


def test_choice_counts_the_correction_and_weights_do_not():
    h, w = torch.randn(20, 8, dtype=O.F64), torch.randn(5, 8, dtype=O.F64)
    s = torch.softmax(h @ w.t(), -1)
    idx, wt = O.route(h, w, torch.tensor([0.0, 0, 0, 0, 9.0]), 2)
    assert (idx[:, 0] == 4).all() and torch.allclose(wt[:, 0], s[:, 4]) and (wt.sum(-1) < 1).all()


def test_identity_experts_pass_the_input_on():
    cfg = M.moe(1, 1, 4, 1, 0)
    h = torch.randn(9, 6, dtype=O.F64)
    w = {"router": torch.randn(2, 6, dtype=O.F64), "correction": torch.tensor([0.0, 5.0]), "e0.gate": torch.randn(4, 6), "e0.up": torch.randn(4, 6), "e0.down": torch.randn(6, 4)}
    assert torch.allclose(O.moe_ff(h, lambda n: w[n].double(), cfg), torch.softmax(h @ w["router"].t(), -1)[:, 1:] * h)


def test_a_later_token_changes_nothing_before_it():
    cfg = M.small()
    w = M.weights(cfg, 5)
    t = M.tokens(20, cfg["vocab"], 1)
    a, b = O.forward(cfg, w, t), O.forward(cfg, w, t[:12] + M.tokens(8, cfg["vocab"], 2))
    assert torch.allclose(a[:12], b[:12]) and not torch.allclose(a[12:], b[12:])


# -- configuration, names, files --------------------------------------------------------------------------------
@pytest.mark.parametrize("base,dims,s", [(800.0, 12, M.YARN), (1e4, 128, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}), (50.0, 4, {"factor": 2.0, "original": 10, "fast": 40.0, "slow": 20.0})])
def test_rotation_with_a_ramp_over_the_pairs(base, dims, s):
    r = Rotation(dims, base, None, False, (s["factor"], s["original"], s["fast"], s["slow"]))
    want, c = O.yarn_freqs(base, dims, **s)
    assert torch.allclose(torch.tensor(r.freqs(), dtype=torch.float64), want, rtol=1e-13) and r.magnitude == pytest.approx(c) == pytest.approx(0.1 * math.log(s["factor"]) + 1)
    ratio = want / torch.tensor(Rotation(dims, base).freqs(), dtype=torch.float64)
    assert ratio.max() <= 1 + 1e-12 and ratio.min() >= 1 / s["factor"] - 1e-12 and (ratio[1:] <= ratio[:-1] + 1e-12).all()


def test_configuration():
    st = parse_stack(M.small())
    assert [type(L.mixer) for L in st.layers] == [AttentionMixer, Mamba2Mixer, AttentionMixer, Mamba2Mixer, AttentionMixer, AttentionMixer]
    assert [type(L.mlp) for L in st.layers] == [ExpertMLP, type(None), ExpertMLP, ExpertMLP, type(None), type(None)]
    a, f = st.layers[0].mixer, st.layers[2].mixer
    assert (a.window, a.keep, a.chunk, a.conv, a.gate, a.qk_norm, a.bias, a.keys_as_values, a.n_gate, a.n_v) == (37, 3, 0, 4, "element", "head", "", False, 4 * 28, 2 * 28)
    assert (f.window, f.keep, f.conv, f.gate, f.bias, f.keys_as_values, f.n_gate, f.n_v) == (0, 0, 0, "head", "qk", True, 6, 0)
    assert a.rot.yarn == (3.0, 90.0, 9.0, 0.7) and a.rot.scaling is None and f.rot.scaling == (5.0, 1.0, 3.5, 70.0) and f.rot.magnitude == 1.0
    e = st.layers[0].mlp
    assert (e.experts, e.top, e.identity, e.outputs, e.act, e.scoring, e.router_bias, e.correction, e.shared_gate) == (6, 3, 2, 8, "silu", "all", False, True, True)
    assert st.layers[2].mlp.shared is None and st.layers[3].mlp.top == 4
    assert st.logit_scale == 0.37 and st.design.post_norm and st.recurrent and not st.design.parallel
    kv = [2 * (20 + 28), 3 * 48, 1 * (16 + 40), 4 * 60]
    conv = [(4 * 20 + 2 * 48) * 3, (3 * 16 + 16 + 40) * 1]
    state = [60 * 9 + (60 + 18) * 1, 72 * 20 + (72 + 120) * 2]
    assert st.kv_bytes_per_token() == 2 * sum(kv) and st.state_bytes() == 4 * (sum(conv) + sum(state))
    assert not parse_stack(M.config([M.full()])).recurrent and parse_stack(M.config([M.windowed()])).recurrent and not parse_stack(M.config([M.windowed(conv=1)])).recurrent


def test_bad_configurations_are_refused():
    for change in (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), lambda c: c["layers"][0].update(type="mamba3"), lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
                   lambda c: c["layers"][1]["mixer"].update(norm_groups=7), lambda c: c["layers"][3]["mixer"].update(groups=4), lambda c: c["layers"][2]["mixer"].update(vdim=25),
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
        assert ca.stack == cb.stack == parse_stack(cfg) and ca.recurrent and ca.arch == "tirudra" and ca.vocab_size == cfg["vocab"] and ca.n_experts == 6
        assert set(a.tensors) == set(b.tensors)
        for n in a.tensors:
            x, y = load_tensor(a, n), load_tensor(b, n)
            assert x.shape == y.shape and torch.equal(x.dequant(), y.dequant()), n

        def get(n):
            return load_tensor(b, n).dequant()
        for gg, n in (("attn_norm", "norm1"), ("ffn_norm", "norm2"), ("post_attention_norm", "norm1b"), ("post_ffw_norm", "norm2b")):
            assert torch.equal(get(f"blk.0.{gg}.weight"), w[f"l0.{n}"].float() + 1)
        assert torch.equal(get("blk.0.attn_q_norm.weight"), w["l0.mix.q.norm"].float()) and torch.equal(get("blk.1.ssm_norm.weight"), w["l1.mix.norm"].float())
        assert torch.equal(get("blk.1.ssm_out.weight"), w["l1.mix.o"].float()) and torch.equal(get("blk.0.attn_q_conv1d.weight"), w["l0.mix.q.conv"].float())
        assert torch.allclose(get("blk.1.ssm_a"), -torch.exp(w["l1.mix.A_log"].double()).float())
        assert torch.equal(get("blk.0.ffn_up_exps.weight"), torch.stack([w[f"l0.mlp.e{e}.up"].float() for e in range(6)]))
        assert torch.equal(get("blk.0.exp_probs_b.bias"), w["l0.mlp.correction"].float()) and torch.equal(get("blk.0.ffn_gate_inp_shexp.weight"), w["l0.mlp.shared.sg"].float())
        with pytest.raises(NotImplementedError):
            make_backend(a, "cpu")


def test_missing_and_unknown_tensors_are_errors(tmp_path):
    cfg = M.small()
    for name, change in (("l0.mlp.e5.up", "drop"), ("l0.mix.extra", "add"), ("l0.mlp.e6.up", "add")):
        w = M.weights(cfg, 3)
        if change == "drop":
            del w[name]
        else:
            w[name] = torch.zeros(3, 3, dtype=torch.bfloat16)
        with pytest.raises(ValueError):
            open_model(M.write(tmp_path / name, cfg, w))


def test_memory_estimate_counts_cache_and_state():
    from ollama_b200.convert.stack import stack_kv
    from ollama_b200.server.sched import predict_memory

    class Model:
        size = 1000

        def kv(self):
            return stack_kv(M.small(), "m")
    st = parse_stack(M.small())
    assert predict_memory(Model(), 100, 2) == 1000 + 2 * (100 * st.kv_bytes_per_token() + st.state_bytes())


def test_synthetic_models_have_every_tensor():
    from ollama_b200.models.synth import STACK_SPECS, SyntheticStackTensors
    cfg = STACK_SPECS["tiny-tirudra"]
    t = SyntheticStackTensors(cfg)
    from ollama_b200.convert.stack import map_stack_name
    assert set(t.keys()) == {map_stack_name(n, cfg) for n in M.shapes(cfg)}


# -- scheduler and trace replay over a stand-in back end -----------------------------------------------------------
class Plain(V.Plain):
    def __init__(self, cfg, w):
        super().__init__(cfg, w)
        self.cfg = ModelConfig(arch="tirudra", vocab_size=cfg["vocab"], stack=parse_stack(cfg))

    def step(self, segs, want):
        self.calls.append([len(t) for _, t, _ in segs])
        out = []
        for (slot, toks, p0), rows in zip(segs, want):
            self.cache.reserve(slot, p0 + len(toks))
            if p0 == 0:
                self.seen[slot] = []
            assert len(self.seen[slot]) == p0, "a recurrent state was asked to move back"
            self.seen[slot] = self.seen[slot] + list(toks)
            if len(rows):
                lg = O.forward(self.raw, self.w, self.seen[slot], torch.float32)
                out += [lg[p0 + r] for r in rows]
        return torch.stack(out) if out else None


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(cfg, w, seq, torch.float32)[-1].argmax()))
    return seq[len(prompt):]


@pytest.fixture(scope="module")
def tiny():
    cfg = M.config([M.windowed(M.moe(3, 2, 8, 1, 6), size=9, keep=2), M.mamba(heads=2, vdim=4, state=6, groups=1), M.full(heads=2, kv_heads=1, dim=8, rot={"base": 50.0, "dims": 8})], width=24, vocab=61)
    return cfg, M.weights(cfg, 5)


def test_scheduler_mixes_prompts_waits_for_pages_and_reuses_a_prefix_only_as_a_whole(tiny):
    cfg, w = tiny
    be = Plain(cfg, w)
    r = Runner(None, RunnerOptions(num_ctx=2 * PAGE, num_parallel=3, num_batch=9, kv_pool_tokens=3 * PAGE), backend=be)

    def submit(p, n):
        return r.submit(CompletionRequest(prompt=p, sampling=SamplingParams(temperature=0), num_predict=n, ignore_eos=True))
    try:
        prompts = [M.tokens(n, cfg["vocab"], n) for n in (3, 66, 18, 9)]
        seqs = [submit(p, 4) for p in prompts]
        assert [V.drain(s)[0] for s in seqs] == [greedy(cfg, w, p, 4) for p in prompts]
        assert any(1 in c and max(c) > 1 for c in be.calls)
        p = M.tokens(20, cfg["vocab"], 1)
        out, _ = V.drain(submit(p, 4))
        longer = p + out[:-1] + M.tokens(5, cfg["vocab"], 2)
        got, ch = V.drain(submit(longer, 3))
        assert ch.cached_tokens == len(p) + 3 and got == greedy(cfg, w, longer, 3)
        branch = p[:12] + M.tokens(9, cfg["vocab"], 3)
        got, ch = V.drain(submit(branch, 3))
        assert ch.cached_tokens == 0 and got == greedy(cfg, w, branch, 3)
    finally:
        r.close()


def test_replay_of_a_trace(tiny, tmp_path):
    import numpy as np
    cfg, w = tiny
    be = Plain(cfg, w)
    be.alloc(4, 128, 256)
    a = M.tokens(9, cfg["vocab"], 1)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:4], "want": [1, 3]}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": a[4:], "want": [4]}], "end": ["x"]}]
    said = []
    replay(be, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    full = O.forward(cfg, w, a).float().numpy()
    assert said == ["done 0", "done 1"]
    assert np.allclose(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1), full[[1, 3]], atol=1e-4)
    assert np.allclose(np.fromfile(tmp_path / "1.f32", "<f4"), full[8], atol=1e-4)
    assert len(be.cache.free) == be.cache.n_pages
