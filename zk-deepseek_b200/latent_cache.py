"""Cache of the latent-attention layers of a floating-point decoder: per position one normed latent and one rotated
key part, shared by all heads.

A request holds one slot, `capacity` positions long, in the buffer of every layer that has a key/value projection of
its own; a layer that reads another layer's latents has no buffer and is pointed at that layer's.  Buffers are zeroed
once: what a released slot leaves behind is finite, is never visible to the next request (its mask ends at its own
position) and is overwritten as that request grows.
"""
import torch


class CacheFull(RuntimeError):
    """no free slot, or a request longer than a slot"""


class LatentCache:
    def __init__(self, pitches, owners, slots, capacity, dtype, device):
        """pitches: row pitch (elements) of every layer that stores latents, None for the others;
        owners: for every layer the layer whose buffer it reads"""
        self.slots, self.capacity = slots, capacity
        self.owners = list(owners)
        self.buffers = [None if p is None else torch.zeros(slots, capacity, p, dtype=dtype, device=device)
                        for p in pitches]
        for i, o in enumerate(self.owners):
            if o is not None and self.buffers[o] is None:
                raise ValueError("layer %d reads the latents of layer %d, which stores none" % (i, o))
        self._free = list(range(slots - 1, -1, -1))
        self.lengths = [0] * slots

    def buffer(self, layer):
        return self.buffers[self.owners[layer]]

    def acquire(self):
        if not self._free:
            raise CacheFull("all %d cache slots are in use" % self.slots)
        slot = self._free.pop()
        self.lengths[slot] = 0
        return slot

    def release(self, slot):
        if slot in self._free or not 0 <= slot < self.slots:
            raise ValueError("slot %d is not in use" % slot)
        self.lengths[slot] = 0
        self._free.append(slot)

    def extend(self, slot, start, n):
        """the step about to run writes positions start .. start + n - 1 of the slot"""
        if start != self.lengths[slot]:
            raise ValueError("slot %d holds %d positions, the step starts at %d" % (slot, self.lengths[slot], start))
        if start + n > self.capacity:
            raise CacheFull("%d positions do not fit a slot of %d" % (start + n, self.capacity))
        self.lengths[slot] = start + n

    def truncate(self, slot, length):
        """forget the positions from `length` on"""
        if not 0 <= length <= self.lengths[slot]:
            raise ValueError("slot %d holds %d positions" % (slot, self.lengths[slot]))
        self.lengths[slot] = length

    def free_slots(self):
        return len(self._free)

    def bytes(self):
        return sum(b.numel() * b.element_size() for b in self.buffers if b is not None)
