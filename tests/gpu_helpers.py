"""Shared by the GPU tests: a step's batch and context without an engine, random operands, comparisons."""
import numpy as np
import torch

STORE = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def up64(n):
    return (n + 63) // 64 * 64


class _Batch:
    pass


class _Ctx:
    def __init__(self, device="cuda:0"):
        from garuda_b200.engine.batch import Workspace
        self.ws = Workspace(torch.device(device))
        self.batch = _Batch()


def rnd(*shape, dtype=torch.float32, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(hash((shape, seed)) % (1 << 31))
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def close(got, want, dt, what, tol=None):
    got, want = got.float().cpu(), want.float()
    tol = tol or (2e-2 if dt == torch.bfloat16 else 2e-5)
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert torch.isfinite(got).all() and err <= tol, f"{what}: {err:.2e}"


def step_batch(lens, starts, slots, page_size, seed=1):
    """A batch of requests that bring ``lens`` tokens from positions ``starts``, their pages drawn at
    random from the pool; returns (batch, block table, pages in the pool)."""
    b = _Batch()
    R = len(lens)
    b.cu_q = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    b.kv_lens = torch.tensor([s + n for s, n in zip(starts, lens)], dtype=torch.int32)
    b.positions = torch.tensor(np.concatenate([np.arange(s, s + n) for s, n in zip(starts, lens)]), dtype=torch.int32)
    b.slots = torch.tensor(slots, dtype=torch.int32)
    b.token_req = torch.repeat_interleave(torch.arange(R, dtype=torch.int32), torch.tensor(lens))
    b.num_requests, b.max_q_len, b.min_q_len = R, max(lens), min(lens)
    b.num_tokens, b.max_kv_len = sum(lens), int(b.kv_lens.max())
    width = (b.max_kv_len + page_size - 1) // page_size + 1
    table = -torch.ones(R, width, dtype=torch.int32)
    perm = np.random.default_rng(seed).permutation(R * width)
    at = 0
    for r in range(R):
        n = (int(b.kv_lens[r]) + page_size - 1) // page_size
        table[r, :n] = torch.tensor(perm[at:at + n], dtype=torch.int32)
        at += n
    return b, table, R * width


def batches(b):
    ctx_g, ctx_r = _Ctx(), _Ctx("cpu")
    ctx_r.batch = b
    bg = _Batch()
    for k, v in vars(b).items():
        setattr(bg, k, v.cuda() if torch.is_tensor(v) else v)
    ctx_g.batch = bg
    return ctx_g, ctx_r
