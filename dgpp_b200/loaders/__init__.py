# Families with a published checkpoint layout of their own; they run in bf16 and in true fp32.  (Here, because the trace replay asks
# before the host runtime is built.)
PUBLISHED = ("sitirax", "potivik", "vevapel", "tefudra")
