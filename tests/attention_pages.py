"""A paged key/value cache filled by hand, for the tests of the attention kernels."""
import torch

DEV = torch.device("cuda:0")


class Pages:
    """A hand-made paged cache whose pages are handed out in a scrambled order and start as NaN; pages no
    token of position ``from_pos`` on may read are taken away before a step (as the cache does)."""

    def __init__(self, n_slots, max_len, n_kv, d, dv, dt, window, keep, seed=0):
        from builderforce_inference_b200.cache import KVView
        blocks = (max_len + 63) // 64
        n_pages = n_slots * blocks + 3
        perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
        self.window, self.keep = window, keep
        self.table = torch.tensor(perm[:n_slots * blocks], dtype=torch.int32).reshape(n_slots, blocks)
        self.k = torch.full((n_pages, n_kv, 64, d), float("nan"), dtype=dt, device=DEV)
        self.v = torch.full((n_pages, n_kv, 64, dv), float("nan"), dtype=dt, device=DEV)
        self.view = KVView(self.k, self.v, self.table.to(DEV), n_kv, d, window, v_dim=None if dv == d else dv, keep_first=keep)

    def write(self, slot, k, v):
        n = k.shape[0]
        pad = (-n) % 64
        nan = float("nan")
        for store, x in ((self.k, k), (self.v, v)):
            x = torch.cat([x, torch.full((pad,) + tuple(x.shape[1:]), nan)]) if pad else x
            x = x.reshape(-1, 64, x.shape[1], x.shape[2]).permute(0, 2, 1, 3).to(store.dtype).to(DEV)
            store[self.table[slot, :x.shape[0]].long().to(DEV)] = x

    def forget(self, starts):
        """Before a step in which slot s goes on at position starts[s]: pages nothing will read again."""
        dev = self.table.clone()
        for slot, start in starts.items():
            first = max(0, start - self.window + 1) // 64 if self.window else 0
            dev[slot, (self.keep + 63) // 64:first] = -1
        self.view.block_table = dev.to(DEV)
