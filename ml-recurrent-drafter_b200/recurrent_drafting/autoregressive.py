"""One-token-per-step decoding over the same models, caches and kernels
(recurrent_drafting/autoregressive.py:13-53).  The comparator of the speculative loop: with greedy
search both must produce the same tokens.

As in the reference, a Llama token's position is its column index in the left-padded input (the
reference passes arange(past, cur) without subtracting the padding, autoregressive.py:37-39); models
whose positions count from each sequence's first token (positions_are_columns = False) store their
rows without the padding."""
from typing import Generator, Optional

import torch

from . import _lib
from .recurrent_drafting import SamplingArgs, SpecialTokens, _count_left_paddings
from .session import DecodeGraphs, Session, graphs_enabled


@torch.inference_mode()
def generate(model, input_ids: torch.Tensor, max_length: int, special_tokens: SpecialTokens,
             sampling_args: SamplingArgs = SamplingArgs(1.0, True),
             cuda_graphs: Optional[bool] = None) -> Generator[torch.Tensor, None, None]:
    """Yields the (batch, length) token matrix after every step.  model: a RecurrentDrafting, or a base model of the
    registry.  Steps after the second are replayed from CUDA graphs where the model allows it."""
    llm = getattr(model, "llm", model)
    B, Lp = input_ids.shape
    dev = input_ids.device
    if not input_ids.is_cuda:
        raise _lib.RedrafterError("input_ids must live on a CUDA device: this package has no CPU path")
    pads = _count_left_paddings(input_ids, special_tokens.pad)
    live = torch.arange(Lp, device=dev)[None, :] >= pads[:, None]
    first = pads.tolist()
    assert max(first) < Lp, "a prompt row holds only padding"
    session = Session(llm, B, max_length, begin=first if llm.positions_are_columns else None)
    tok_ids = input_ids[live].contiguous()
    counts = [Lp - p for p in first]
    hidden = session.extend(tok_ids, counts)
    ends = torch.cumsum(torch.tensor(counts), 0).sub_(1).to(dev)
    session.last_hidden.copy_(hidden[ends])
    tokens = torch.full((B, max_length), special_tokens.pad, dtype=torch.int64, device=dev)
    tokens[:, :Lp] = input_ids
    columns = pads.to(torch.int32)
    use_graphs = graphs_enabled(llm, cuda_graphs)
    graphs: Optional[DecodeGraphs] = None
    length = Lp
    steps = 0
    while length < max_length:
        if use_graphs and graphs is None and steps == 2:
            graphs = DecodeGraphs(session, sampling_args, tokens, columns)
        steps += 1
        if not sampling_args.greedy:
            session.draw_uniforms()
        if graphs is not None:
            graphs.pick.replay()
            _lib.count_replay(graphs.n_pick)
        else:
            session.pick(sampling_args, tokens, columns)
        length += 1
        out = tokens[:, :length].clone()
        yield out
        if special_tokens.eos is not None and bool(((out[:, Lp:] == special_tokens.eos).sum(dim=-1) > 0).sum() == B):
            break
        if length >= max_length:
            break
        if graphs is not None:
            graphs.forward.replay()
            _lib.count_replay(graphs.n_forward)
        else:
            session.forward(session.max_length if use_graphs else length)
    session.check()
