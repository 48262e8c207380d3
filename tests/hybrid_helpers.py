"""What the GPU tests of the hybrid designs share: batches of portions, comparison with the plain
implementation, a mixer or a model run in portions."""

import pytest
import torch

from llm_compiler_b200 import hybrid_kernels as hk
from llm_compiler_b200 import kernels


EPS = 1e-5
TOLERANCE = {torch.float32: 3e-5, torch.bfloat16: 3e-2}


def batch_of(portions):
    """SequenceBatch of (slot, first position, count) portions."""
    counts = [count for _, _, count in portions]
    starts = [sum(counts[:i]) for i in range(len(counts) + 1)]
    vector = lambda values: torch.tensor(values, dtype=torch.int32, device="cuda")
    return hk.SequenceBatch(starts[-1], len(portions),
                            vector([i for i, c in enumerate(counts) for _ in range(c)]), vector(starts),
                            vector([slot for slot, _, _ in portions]), vector([base for _, base, _ in portions]),
                            counts, [base for _, base, _ in portions], [slot for slot, _, _ in portions])


def close(actual, expected, dtype, factor=1.0):
    """Root mean square error per row, relative to the largest row."""
    actual, expected = actual.double().cpu(), expected.double()
    error = (actual - expected).pow(2).mean(-1).sqrt()
    scale = expected.pow(2).mean(-1).sqrt().max()
    worst = float((error / scale).max())
    assert worst <= TOLERANCE[dtype] * factor, f"relative error {worst} at row {int(error.argmax())}"


def summed(y):
    """A sublayer's result in one piece, as residual_norm adds it up."""
    if isinstance(y, hk.Summands):
        total = 0.0 if y.y is None else summed(y.y)
        if y.bias is not None:
            total = total + torch.nn.functional.pad(y.bias.float(), (0, total.shape[1] - y.bias.shape[0]))
        return total if y.rows is None else total + y.rows.float()[y.places.long()].sum(1)
    return y.sum(0) if y.ndim == 3 else y.float()


def run_mixer(mixer, h, cuts, *, slot=1, slots=3, capacity=512, state=None, garbage=True):
    """The mixer's rows for one sequence, run in portions of the given sizes."""
    if state is None:
        state = {name: torch.zeros((slots, *shape), dtype=dtype, device="cuda")
                 for name, (shape, dtype) in mixer.state_spec(capacity).items()}
        if garbage:  # what a former sequence left: nothing of it may be read
            for tensor in state.values():
                tensor.fill_(3.0)
    rows, first = [], 0
    for cut in cuts:
        piece = torch.zeros((cut, hk.pad8(h.shape[1])), dtype=h.dtype, device="cuda")
        piece[:, :h.shape[1]] = h[first:first + cut].cuda()
        rows.append(summed(mixer(piece, batch_of([(slot, first, cut)]), state))[:, :h.shape[1]])
        first += cut
    kernels.runtime().check_status()
    return torch.cat(rows)


def random_rows(tokens, width, dtype, seed):
    return torch.randn(tokens, width, generator=torch.Generator().manual_seed(seed)).to(dtype)


def cuda(weights):
    return {name: w.cuda() for name, w in weights.items()}


def double(weights):
    return {name: w.double() for name, w in weights.items()}


CUTS = [[150], [1] * 150, [2, 3, 61, 64, 20], [63, 2, 65, 2, 18], [128, 22], [7, 1, 1, 1, 90, 50]]
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])


def tokens_of(config, count, seed):
    return torch.randint(0, config.vocab_size, (count,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cut(engine, tokens, cuts):
    slot, rows, first = engine.open(), [], 0
    for cut in cuts:
        rows.append(engine.forward([(slot, tokens[first:first + cut])], [list(range(cut))]))
        first += cut
    engine.state.check()
    engine.close(slot)
    return torch.cat(rows)


# A single row of a bf16 model may sit where a small read-out is normed to size one and its rounding
# errors with it (the same row passes in fp32): the worst row gets more room than a mechanism alone.
MODEL_TOLERANCE = {torch.float32: 1.0, torch.bfloat16: 5.0}
