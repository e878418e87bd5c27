"""Helpers of the decoder-model tests: hand-made step layouts, replay of schedules through an engine, error measures."""
import torch

DEV = "cuda:0"


class Lay:
    """A hand-made step layout for kernel tests: sequences [(pos0, n_new, block_table)]; n_new 0 is a padding row."""

    def __init__(self, seqs, page, max_blocks):
        tok_seq, pos, slots, start, o = [], [], [], [], 0
        for b, (p0, n, bt) in enumerate(seqs):
            start.append(o)
            for t in range(max(n, 1)):
                p = p0 + t
                tok_seq.append(b), pos.append(p), slots.append(bt[p // page] * page + p % page if n else -1)
            o += max(n, 1)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        self.tok_seq, self.positions, self.slot_mapping = i32(tok_seq), i32(pos), i32(slots)
        self.seq_start, self.seq_pos0 = i32(start), i32([s[0] for s in seqs])
        self.seq_len, self.seq_slot = i32([s[1] for s in seqs]), i32(list(range(len(seqs))))
        bt = torch.zeros(len(seqs), max_blocks, dtype=torch.int32)
        for b, s in enumerate(seqs):
            bt[b, :len(s[2])] = torch.tensor(s[2], dtype=torch.int32)
        self.block_tables = bt.to(DEV)
        self.n_tokens, self.n_seqs, self.max_new = o, len(seqs), max(s[1] for s in seqs)


def rel(a, b):
    return ((a.double().cpu() - b.double().cpu()).abs().max() / b.double().abs().max().clamp_min(1e-30)).item()


def make_engine(config, sd: dict, dtype="float32", pages=12, page=64, seqs=4, slots=None, eager=True, budget=None, max_len=256):
    from nano_qwen3tts_vllm_b200.engine.llm_engine.lm_engine import CausalLMEngine
    return CausalLMEngine(config, state_dict={k: v.to(torch.bfloat16) for k, v in sd.items()}, dtype=dtype, kvcache_block_size=page,
                          num_kvcache_blocks=pages, max_num_seqs=seqs, max_state_slots=slots or seqs, max_model_len=max_len,
                          max_num_batched_tokens=budget or seqs * max_len, enforce_eager=eager, device=DEV)


def replay(engine, requests: dict, schedule: list):
    """Feed ``schedule`` = [[(id, count), ...], ...] through engine.step as held sequences; logits of every position."""
    at = {i: 0 for i in requests}
    live, got = set(), {i: [] for i in requests}
    for step in schedule:
        want = {}
        for i, n in step:
            toks = requests[i][at[i]:at[i] + n]
            if i in live:
                engine.feed(i, toks)
            else:
                engine.add_request(toks, request_id=i, hold=True)
                live.add(i)
            want[i] = list(range(n))
            at[i] += n
        out = engine.step(want=want)
        assert out.scheduled == {i: n for i, n in step}
        o = 0
        for i, n in step:
            got[i].append(out.logits[o:o + n].double().cpu())
            o += n
        for i, _ in step:
            if at[i] == len(requests[i]):
                engine.clear_request(i)
                live.discard(i)
    return {i: torch.cat(v) for i, v in got.items() if v}


def nerr_rows(got, ref):
    """Per-position error: rms over the vocabulary of the mean-free difference, relative to the rms of the logits."""
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()


def nerr(got, ref):
    return nerr_rows(got, ref).max().item()


def tokens_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def cuts_of(T, sizes=(2, 3, 1, 17, 2, 1, 1, 30, 2)):
    """Portions of changing size, then single tokens."""
    cuts, left = [], T
    for n in sizes:
        n = min(n, left)
        if n:
            cuts.append(n)
            left -= n
    return cuts + [1] * left
