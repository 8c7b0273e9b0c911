"""What the GPU tests of mixer parts share: tensors on the device, batches' index arrays, and a harness that
gives one mixer pages and state slots and runs it step by step."""

import torch


def dev(t, dtype=None):
    return t.to("cuda", dtype) if dtype is not None else t.to("cuda")


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device="cuda")


def rel(got, want) -> float:
    got, want = got.detach().double().cpu(), want.double()
    return float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))


def rand(shape, seed):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def batch(lengths):
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    seq = [b for b, n in enumerate(lengths) for _ in range(n)]
    return i32(cu), i32(seq)


class Harness:
    """Pages and state slots for one mixer (and for mixers that read its pages), and steps of
    (sequence, its next n tokens) in any batch; pages come in a shuffled order and freed ones are used again first."""

    def __init__(self, mixer, dtype, page=16, num_pages=96, slots=5, seed=0, readers=()):
        self.mixers, self.dtype, self.page = [mixer, *readers], dtype, page
        need = mixer.cache_need()
        self.k = self.v = None
        if need.kind != "none":
            self.k = torch.full((num_pages, page, *need.k_row), float("nan"), device="cuda", dtype=dtype)
            self.v = None if need.v_row is None else torch.full((num_pages, page, *need.v_row), float("nan"), device="cuda", dtype=dtype)
        self.states = [None if m.cache_need().state_shape is None else torch.zeros((slots, *m.cache_need().state_shape), device="cuda")
                       for m in self.mixers]
        self.free_pages = torch.randperm(num_pages, generator=torch.Generator().manual_seed(seed)).tolist()
        self.pages, self.done, self.slot = {}, {}, {}
        self.free_slots = list(range(slots))[::-1]

    def end(self, name):
        self.free_pages = self.pages.pop(name, []) + self.free_pages
        self.free_slots.append(self.slot.pop(name))
        del self.done[name]

    def step(self, x_by_seq, which=0):
        """Runs mixer `which` (0: the one that fills the pages) on the given rows; a reader runs on positions that
        the writer has stored already (`advance` False then)."""
        from tokensprint_b200 import ops
        from tokensprint_b200.parts.base import GroupTables, LayerCache, StepContext

        names = sorted(x_by_seq, key=lambda n: (x_by_seq[n].shape[0] != 1, n))  # single tokens first, as the runner orders them
        pos, seq, cu, ctx, slots, slot_map, rows = [], [], [0], [], [], [], []
        for b, name in enumerate(names):
            n = x_by_seq[name].shape[0]
            if name not in self.done:
                self.done[name], self.pages[name] = [0] * len(self.mixers), []
                self.slot[name] = self.free_slots.pop()
                for st in self.states:
                    if st is not None:
                        st[self.slot[name]].zero_()
            start = self.done[name][which]
            while len(self.pages[name]) * self.page < start + n:
                self.pages[name].append(self.free_pages.pop(0))
            pos += range(start, start + n)
            seq += [b] * n
            cu.append(cu[-1] + n)
            ctx.append(start + n)
            slots.append(self.slot[name])
            slot_map += [self.pages[name][p // self.page] * self.page + p % self.page for p in range(start, start + n)]
            rows.append(x_by_seq[name])
            self.done[name][which] = start + n
        width = max(len(self.pages[n]) for n in names)
        table = [self.pages[n] + [-1] * (width - len(self.pages[n])) for n in names]
        T = cu[-1]
        lens = [x_by_seq[n].shape[0] for n in names]
        step = StepContext(num_tokens=T, num_seqs=len(names), token_ids=i32([0] * T), positions=i32(pos), seq_index=i32(seq),
                           cu_seqlens_q=i32(cu), context_lens=i32(ctx), state_slots=i32(slots),
                           groups=[GroupTables(i32(sum(table, [])).view(len(names), width), i32(slot_map))], page_size=self.page,
                           max_seqlen_q=max(lens), max_context_len=max(ctx), decode_only=all(n == 1 for n in lens),
                           decode_seqs=sum(1 for n in lens if n == 1))
        cache = LayerCache(group=0 if self.k is not None else -1, k_pages=self.k, v_pages=self.v, state=self.states[which], writes=which == 0)
        out = self.mixers[which].forward(dev(torch.cat(rows).to(self.dtype)), step, cache)
        ops.flush_gemm_chain()
        return {name: out[cu[b]:cu[b + 1]].float().cpu() for b, name in enumerate(names)}


def inputs(T, width, seed, dtype):
    return rand((T, width), seed).to(dtype).float()  # what both sides read


def in_portions(h, name, x, sizes, which=0):
    out, pos, i = [], 0, 0
    while pos < x.shape[0]:
        n = min(sizes[i % len(sizes)], x.shape[0] - pos)
        out.append(h.step({name: x[pos:pos + n]}, which)[name])
        pos, i = pos + n, i + 1
    return torch.cat(out)
