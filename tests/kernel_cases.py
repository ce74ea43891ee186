"""Set-up shared by the tests that run single kernels: an op set without a model, random tensors, comparison with fp64, and a
state whose pages are scattered."""
import types

import torch

from phaseshift_b200.runtime.batch import SeqRows, StepBatch
from phaseshift_b200.runtime.state import ModelState, StateConfig

BF, F32 = torch.bfloat16, torch.float32


def ops_of(dtype=BF, max_len=2048):
    from phaseshift_b200.ops.cuda_ops import CudaOps
    return CudaOps(types.SimpleNamespace(), torch.device("cuda:0"), max_seq_len=max_len, act_dtype=dtype)


def rnd(*shape, seed=0, scale=1.0, dtype=F32):
    g = torch.Generator(device="cuda").manual_seed(seed)
    return (torch.randn(shape, device="cuda", generator=g) * scale).to(dtype)


def close(got, want, tol):
    d = (got.double() - want.double()).abs().max()
    assert float(d) <= tol * max(1e-6, float(want.double().abs().max())), float(d)


class Paged:
    """One layer run: a state with scattered pages for sequences of given lengths and a step batch over their last rows."""

    def __init__(self, spec, seqs, dtype, page=16, graph=False):
        self.seqs = seqs                                   # [(first position of the step, rows of the step)]
        longest = max(p + n for p, n in seqs)
        cfg = types.SimpleNamespace(geometry=lambda r, s: None, state_specs=lambda g: [spec])
        sc = StateConfig(max_slots=len(seqs) + 1, max_seq_len=longest + 5, page_tokens=page)
        self.st = ModelState(cfg, sc, torch.device("cuda:0"), dtype)
        rows = sum(n for _, n in seqs)
        self.b = StepBatch(rows + 3, len(seqs), torch.device("cuda:0"))
        self.b.max_context = longest + 6
        g = torch.Generator().manual_seed(5)
        pages = (torch.randperm(self.st.num_pages - 1, generator=g) + 1).tolist()
        for i, (p, n) in enumerate(seqs):
            for blk in range(-(-(p + n) // page)):
                self.st.block_table[i + 1, blk] = pages.pop()
        self.b.fill([SeqRows(i + 1, p, [0] * n) for i, (p, n) in enumerate(seqs)])
        self.b.graph_static = graph
        self.b.upload()
        self.page, self.rows = page, rows + 3              # three padding rows at the end

    def fill_keys(self, i, k, v=None):
        """Key (and value) rows [n, heads, D] of sequence i from position 0 on."""
        t = torch.arange(k.shape[0], device="cuda")
        pg = self.st.block_table[i + 1][t // self.page].long()
        self.st.kv[0].k[pg, :, t % self.page] = k.to(self.st.kv[0].k.dtype)
        if v is not None:
            self.st.kv[0].v[pg, :, t % self.page] = v.to(self.st.kv[0].v.dtype)
