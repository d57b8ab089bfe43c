"""The Rinirax design without a GPU: its plain implementation, configuration, converter, directory reader, and the scheduler with a stand-in
back end that computes with the plain implementation."""
import io
import json
import math

import pytest
import torch

import rinirax_models as M
import rinirax_oracle as O
import test_vazatar_cpu as V
from ollama_b200.convert.hf import convert_hf
from ollama_b200.engine.backend import make_backend, open_model
from ollama_b200.engine.cache import PAGE
from ollama_b200.engine.runner import CompletionRequest, Runner, RunnerOptions
from ollama_b200.engine.sampler import SamplingParams
from ollama_b200.engine.trace import replay
from ollama_b200.models.config import ModelConfig, config_from_gguf
from ollama_b200.models.stack import AttentionMixer, DenseMLP, ExpertMLP, GruMixer, LatentMixer, parse_stack
from ollama_b200.models.weights import load_tensor


def r64(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed), dtype=O.F64)


# -- the plain implementation against identities it must satisfy ------------------------------------------------
def test_layer_norm():
    x, w, b = r64(3, 7), r64(7, seed=1), r64(7, seed=2)
    assert torch.allclose(O.layer_norm(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (7,), w, b, 1e-3))


def test_rotation_of_neighbours_depends_on_distance_only():
    f = O.rotation({"base": 50.0, "dims": 6})[0]
    q, k = r64(1, 1, 9), r64(1, 1, 9, seed=1)

    def at(v, p):
        return O.rotate_pairs(v, torch.tensor([p]), f)[0, 0]
    assert torch.allclose(at(q, 11) @ at(k, 4), at(q, 107) @ at(k, 100)) and not torch.allclose(at(q, 11) @ at(k, 4), at(q, 12) @ at(k, 4))
    assert torch.equal(at(q, 5)[6:], q[0, 0, 6:]) and torch.allclose(at(q, 5)[:2].norm(), q[0, 0, :2].norm())


def test_differential_heads():
    a = r64(4, 3, 8)
    same = O.diff_combine(a, a, 0.25, 0.4, 0.0)
    assert torch.allclose((same ** 2).mean(-1), torch.full((4, 3), 0.36, dtype=O.F64)) and torch.allclose(same / same[..., :1], a / a[..., :1])
    w = {"lq1": torch.zeros(5), "lk1": torch.ones(5), "lq2": torch.ones(5), "lk2": torch.full((5,), -10.0)}
    assert abs(float(O.diff_lambda(lambda n: w[n].double(), 0.3)) - (1.0 - math.exp(-50.0) + 0.3)) < 1e-12


def test_recurrence_is_the_sum_over_earlier_tokens():
    z, u = r64(9, 4), r64(9, 4, seed=1)
    S, g = O.gru_scan(z, u), torch.sigmoid(z)
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    for t in range(9):
        assert torch.allclose(S[t], sum(g[s] * c[s] * (1 - g[s + 1:t + 1]).prod(0) for s in range(t + 1)))
    assert (c > 0).all()


def test_activation_is_smooth_at_zero_and_has_its_slopes():
    z = torch.tensor([-60.0, -1e-6, 0.0, 1e-6, 2.0], dtype=O.F64, requires_grad=True)
    p, q = torch.tensor(0.3, dtype=O.F64), torch.tensor(-0.2, dtype=O.F64)
    y = O.xielu(z, p, q)
    y.sum().backward()
    ap, an = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.2))
    assert torch.allclose(y.detach()[[0, 4]], torch.tensor([an * 59.0 - 30.0, 4 * ap + 1.0], dtype=O.F64))
    assert torch.allclose(z.grad[1:4], torch.full((3,), 0.5, dtype=O.F64), atol=1e-5)


def test_choice_is_made_inside_the_best_groups():
    h = torch.eye(1, 4, dtype=O.F64)
    z = torch.tensor([3.0, -3.0, 1.0, 1.1, 2.0, -9.0], dtype=O.F64)          # groups of two: worth by their two best
    router = torch.zeros(6, 4, dtype=O.F64)
    router[:, 0] = z
    idx, wt = O.route(h, router, torch.zeros(6, dtype=O.F64), 2, 3, 1, 1.5)
    assert sorted(idx[0].tolist()) == [2, 3] and torch.allclose(wt.sum(), torch.tensor(1.5, dtype=O.F64))
    corr = torch.tensor([-5.0, -5.0, -5.0, -5.0, -4.0, -9.0], dtype=O.F64)    # all choice scores negative: what is left out is never chosen
    idx, wt = O.route(h, router, corr, 2, 3, 2, 1.0)
    assert set(idx[0].tolist()) <= {0, 1, 2, 3} and torch.allclose(wt[0], torch.sigmoid(z[idx[0]]) / torch.sigmoid(z[idx[0]]).sum())
    many = r64(50, 4, seed=3)
    full, _ = O.route(many, r64(6, 4, seed=4), torch.zeros(6, dtype=O.F64), 3, 3, 3, 1.0)
    assert torch.equal(full, torch.sigmoid(many @ r64(6, 4, seed=4).t()).topk(3)[1])


def test_depth_average_of_the_last_result_alone_is_a_residual_stream():
    cfg = M.config([M.gru(M.dense()), M.diff(None), M.latent(M.dense())])
    w = M.weights(cfg, 4)
    for i in range(3):
        w[f"l{i}.dwa"] = torch.eye(i + 2)[-1].bfloat16()
    t, x = M.tokens(15, cfg["vocab"], 1), []
    O.forward(cfg, w, t, residuals=x)
    for i in range(3):
        w[f"l{i}.dwa"] = torch.zeros(i + 2).bfloat16()
        w[f"l{i}.dwa"][0] = 1.0
    y = []
    O.forward(cfg, w, t, residuals=y)
    assert all(torch.equal(a, w["embed"].double()[t]) for a in y) and not torch.equal(x[0], x[1])


def test_a_later_token_changes_nothing_before_it():
    cfg = M.small()
    w = M.weights(cfg, 5)
    t = M.tokens(20, cfg["vocab"], 1)
    a, b = O.forward(cfg, w, t), O.forward(cfg, w, t[:12] + M.tokens(8, cfg["vocab"], 2))
    assert torch.allclose(a[:12], b[:12]) and not torch.allclose(a[12:], b[12:])


# -- configuration, names, files --------------------------------------------------------------------------------
def test_configuration():
    st = parse_stack(M.small())
    assert [type(L.mixer) for L in st.layers] == [AttentionMixer, GruMixer, AttentionMixer, LatentMixer, GruMixer, AttentionMixer, LatentMixer, AttentionMixer, GruMixer]
    assert [type(L.mlp) for L in st.layers] == [ExpertMLP, DenseMLP, DenseMLP, ExpertMLP, ExpertMLP] + [type(None)] * 4
    a, s, m = st.layers[0].mixer, st.layers[2].mixer, st.layers[3].mixer
    assert (a.maps, a.diff, a.conv, a.bias, a.qk_norm, a.kv_from, a.n_q, a.n_k, a.n_v, a.gate) == (2, 0.45, 4, "qkv", "", None, 160, 80, 72, "")
    assert (s.kv_from, s.n_q, s.n_k, s.n_v, s.conv) == (0, 160, 0, 0, 2) and a.rot.interleaved and not m.rot.interleaved
    assert (m.window, m.q_rank, m.kv_rank, m.rot.dims, m.rot.yarn) == (37, 44, 36, 12, (3.0, 90.0, 9.0, 0.7)) and m.rot.magnitude == pytest.approx(0.1 * math.log(3.0) + 1.0)
    e = st.layers[0].mlp
    assert (e.experts, e.top, e.groups, e.keep, e.scale, e.scoring, e.correction, e.router_bias, e.act) == (12, 2, 3, 2, 1.7, "sigmoid", True, False, "silu")
    assert st.layers[1].mlp.act == "xielu" and not st.layers[1].mlp.gated
    assert st.design.parallel and st.design.shared_norm and st.design.depth_average and not st.design.paired and st.recurrent
    kv = [2 * (40 + 36), 36 + 12, 36 + 12, 3 * (32 + 16)]
    state = [(160 + 80 + 72) * 3, 70, 160 * 1, 33, 160 * 2, 0, 70]
    assert st.kv_bytes_per_token() == 2 * sum(kv) and st.state_bytes() == 4 * sum(state)
    assert not parse_stack(M.config([M.latent()])).recurrent and not parse_stack(M.config([M.diff(conv=1)])).recurrent and parse_stack(M.config([M.diff()])).recurrent


def test_bad_configurations_are_refused():
    for change in (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=5), lambda c: c["layers"][0].update(type="gru"),
                   lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][2]["mixer"].update(kv_from=2),
                   lambda c: c["layers"][2]["mixer"].update(kv_from=1), lambda c: c["layers"][5]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(dim=24),
                   lambda c: c["layers"][2]["mixer"].update(kv_from=7), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7)):
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
        assert ca.stack == cb.stack == parse_stack(cfg) and ca.recurrent and ca.arch == "rinirax" and ca.vocab_size == cfg["vocab"] and ca.n_experts == 12
        assert set(a.tensors) == set(b.tensors)
        for n in a.tensors:
            x, y = load_tensor(a, n), load_tensor(b, n)
            assert x.shape == y.shape and torch.equal(x.dequant(), y.dequant()), n

        def get(n):
            return load_tensor(b, n).dequant()
        for gg, n in (("blk.0.attn_norm.weight", "l0.norm1"), ("blk.0.attn_norm.bias", "l0.norm1.b"), ("output_norm.bias", "final.norm.b"), ("blk.2.depth_average.weight", "l2.dwa"),
                      ("blk.1.gru_x.weight", "l1.mix.x"), ("blk.1.gru_out.weight", "l1.mix.o"), ("blk.1.ffn_act.weight", "l1.mlp.act"), ("blk.3.attn_q_b.weight", "l3.mix.uq"),
                      ("blk.3.attn_q_a_norm.weight", "l3.mix.dq.norm"), ("blk.0.attn_v.bias", "l0.mix.v.b"), ("blk.0.attn_lambda_k2.weight", "l0.mix.lk2"), ("blk.0.exp_probs_b.bias", "l0.mlp.correction"),
                      ("blk.1.gru_gate.weight", "l1.mix.g")):
            assert torch.equal(get(gg), w[n].float()), gg
        assert torch.equal(get("blk.0.ffn_up_exps.weight"), torch.stack([w[f"l0.mlp.e{e}.up"].float() for e in range(12)]))
        with pytest.raises(NotImplementedError):
            make_backend(a, "cpu")


def test_missing_and_unknown_tensors_are_errors(tmp_path):
    cfg = M.small()
    for name, change in (("l0.mlp.e5.up", "drop"), ("l0.mix.extra", "add"), ("l0.mlp.e12.up", "add")):
        w = M.weights(cfg, 3)
        if change == "drop":
            del w[name]
        else:
            w[name] = torch.zeros(3, 3, dtype=torch.bfloat16)
        with pytest.raises(ValueError):
            open_model(M.write(tmp_path / name, cfg, w))


def test_interleaved_pairs_are_brought_into_the_half_split_order():
    """Queries and keys whose rows are reordered at load give the same scores under the other rotation."""
    from ollama_b200.engine.mixers import HeadAttention
    m = parse_stack(M.config([M.diff(None, heads=2, kv_heads=1, dim=10, rot={"base": 30.0, "dims": 6})])).layers[0].mixer
    holder = HeadAttention.__new__(HeadAttention)
    holder.m = m
    order = holder._half_split(40, "cpu")
    assert sorted(order.tolist()) == list(range(40)) and order[:10].tolist() == [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]
    f, pos = O.rotation({"base": 30.0, "dims": 6})[0], torch.arange(4) * 7
    q, k = r64(4, 40), r64(4, 40, seed=1)
    a, b = (O.rotate_pairs(t.view(4, 4, 10), pos, f) for t in (q, k))
    c, d = (O.rotate_half(t[:, order].view(4, 4, 10), pos, f) for t in (q, k))
    assert torch.allclose(torch.einsum("ihd,jhd->hij", a, b), torch.einsum("ihd,jhd->hij", c, d))


def test_synthetic_models_have_every_tensor():
    from ollama_b200.convert.stack import map_stack_name
    from ollama_b200.models.synth import STACK_SPECS, SyntheticStackTensors
    cfg = STACK_SPECS["tiny-rinirax"]
    assert set(SyntheticStackTensors(cfg).keys()) == {map_stack_name(n, cfg) for n in M.shapes(cfg)}


# -- scheduler and trace replay over a stand-in back end -----------------------------------------------------------
class Plain(V.Plain):
    def __init__(self, cfg, w):
        super().__init__(cfg, w)
        self.cfg = ModelConfig(arch="rinirax", vocab_size=cfg["vocab"], stack=parse_stack(cfg))

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
    cfg = M.config([M.diff(M.moe(4, 2, 8, 2, 1), heads=2, kv_heads=1, dim=8, vdim=12, rot={"base": 50.0, "dims": 6}), M.gru(M.dense(12), width=10), M.latent(None, heads=2, dim=6, rot_dim=4, vdim=8, kv_rank=12, q_rank=8, size=9)], width=24, vocab=61)
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
