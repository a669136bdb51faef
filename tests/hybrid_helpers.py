"""What the tests of hybrid designs share: token ids, the error measure, models around in-memory weights, replayed schedules."""
import torch


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Largest over the positions of rms(difference) / rms(logits), the mean over the vocabulary taken off."""
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return float((d.square().mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).square().mean().sqrt()).max())


def build(cfg, w, dtype, *, max_cached_tokens=1024, max_requests=4, max_sequence_length=512, max_step_tokens=512, cuda_graphs=False,
          **ctx_kw):
    """(model, context, controller) around in-memory weights."""
    from megatron_mixtera_b200 import build as lib
    from megatron_mixtera_b200 import model_registry as R

    lib.build_torch_ops()
    model = R.ARCHITECTURES[cfg["architecture"]](cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, max_sequence_length)
    model.load_checkpoint(w)
    model.config.enable_cuda_graph = cuda_graphs
    ctx = R.make_context(model, max_cached_tokens=max_cached_tokens, max_requests=max_requests, max_step_tokens=max_step_tokens,
                         debug_validate=True, **ctx_kw)
    return model, ctx, R.make_controller(model, ctx)


def replay(controller, schedule, requests):
    """Feed ``schedule`` = [[(request index, count), ...], ...]; a request ends with its last token.  Returns the logits of
    every request at every position."""
    at = {i: 0 for i in range(len(requests))}
    got = {i: [] for i in range(len(requests))}
    for step in schedule:
        entries, want, done, order = [], [], [], []
        for i, n in step:
            part = requests[i][at[i]: at[i] + n]
            assert len(part) == n
            entries.append((i, part))
            want.append(list(range(n)))
            order.append((i, n))
            at[i] += n
            if at[i] == len(requests[i]):
                done.append(i)
        logits = controller.run_given_tokens(entries, want, done).cpu()
        for i, n in order:
            got[i].append(logits[:n])
            logits = logits[n:]
    return {i: torch.cat(v) for i, v in got.items() if v}
