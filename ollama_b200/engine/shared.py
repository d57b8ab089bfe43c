"""Layers of stack models whose mixer and feed-forward read one norm and are added together, x + mixer(norm x) + ff(norm x).

Both parts' first products share a launch where their epilogues allow it, and so do their last ones: W_o a + W_down f is one product over joined columns, also where
f are the chosen experts' columns (a few rows).  The parts are the classes of blocks.py and mixers.py without norms of their own.
"""
from __future__ import annotations

import torch

from ..models.stack import AttentionMixer, DenseMLP, ExpertMLP, GruMixer, LatentMixer, StackLayer
from ..ops import rows as O
from .blocks import DenseFFN, ExpertFFN, GatedRecurrence, LatentAttention, Mat, Step, WeightSource, make_norm, up
from .mixers import HeadAttention


def _mixer(src: WeightSource, p: str, m, f32: bool):
    if isinstance(m, AttentionMixer):
        return HeadAttention(src, p, m, None, f32, None)
    if isinstance(m, LatentMixer):
        return LatentAttention(src, p, m, None, f32)
    if isinstance(m, GruMixer):
        return GatedRecurrence(src, p, m, f32)
    raise NotImplementedError(f"{type(m).__name__} beside a feed-forward that reads the same norm")


class SharedNormLayer:
    def __init__(self, src: WeightSource, p: str, layer: StackLayer, norm: str, f32: bool):
        self.norm = make_norm(src, p + "attn_norm", norm)
        self.mix, self.ff, self.side, self.w_first, self.w_last = _mixer(src, p, layer.mixer, f32), None, None, None, None
        w_in, w_o = self.mix.w_in, self.mix.w_o
        self.mixp = w_o.w.shape[1]
        self.pads = self.mixp != self.mix.n_out          # columns that nobody writes
        if isinstance(layer.mlp, DenseMLP):
            ff = self.ff = DenseFFN(src, p, layer.mlp)
            self.w_last = Mat(torch.cat([w_o.w, ff.down.w], 1))          # the parts' matrices become windows of it
            self.mix.w_o, ff.down = Mat(self.w_last.w[:, :self.mixp]), Mat(self.w_last.w[:, self.mixp:])
        elif isinstance(layer.mlp, ExpertMLP):
            if layer.mlp.shared is not None:
                raise NotImplementedError("a shared expert beside a mixer that reads the same norm")
            ff = self.ff = ExpertFFN(src, p, layer.mlp, None, f32)
            n, bias = w_in.w.shape[0], None
            w = torch.cat([w_in.w, ff.router.w])
            if w_in.bias is not None or ff.router.bias is not None:
                bias = torch.zeros(w.shape[0], device=src.device)
                for at, m in ((0, w_in), (n, ff.router)):
                    if m.bias is not None:
                        bias[at:at + m.bias.numel()] = m.bias
            self.w_first = Mat(w, bias)
            w_in.w, ff.router.w = w[:n], w[n:]

    def run(self, s: Step, mem, h: torch.Tensor) -> None:
        """Adds both parts to the stream; ``h``: its norm."""
        mix, ff = self.mix, self.ff
        if isinstance(ff, ExpertFFN):
            z = s.buf("router", ff.router.w.shape[0], torch.float32)
            if s.small:
                seg = O.seg(ff.router.w, z.shape[1], z, rc=ff.router.bias)
                proj = mix.project(s, h, mem, segs=(seg,))
                ff.mix(s, h, z, beside=mix.w_o, fill=lambda out: mix.mix(s, proj, mem, out))
                return
            if s.act == torch.bfloat16:
                proj = mix.project(s, h, mem, joined=self.w_first, tail=z)
            else:
                proj = mix.project(s, h, mem)
                s.product(h, ff.router, z)
            out = s.buf("mix", self.mixp, zero=self.pads)
            mix.mix(s, proj, mem, out)
            s.add(out, mix.w_o)
            ff.mix(s, h, z)
            return
        cat = s.buf("cat", self.mixp + (ff.ffp if ff else 0), zero=self.pads)
        segs = ()
        if ff is not None:
            f = cat[:, self.mixp:]
            if s.small:
                segs = (O.seg(ff.up.w, ff.ffp, f, act=ff.act, nums=ff.nums),)
            else:
                O.gemm(h, ff.up.w, f, act=ff.act, nums=ff.nums)
                s.launched()
        mix.mix(s, mix.project(s, h, mem, segs=segs), mem, cat[:, :self.mixp])
        s.add(cat, self.w_last if ff is not None else mix.w_o)


class DepthAverage:
    """Weights of the sums over the embedding output and the layers' results: ``w[i]`` of what layer i reads, ``w[-1]`` of the output."""

    def __init__(self, src: WeightSource, n_layers: int):
        one = torch.ones(1, device=src.device)
        self.w = [one, *(src.tensor(f"blk.{i}.depth_average.weight", i + 2).float().contiguous() for i in range(n_layers))]
